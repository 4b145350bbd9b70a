// Short causal convolution over time, one filter per channel, with the last taps-1 inputs of every sequence kept as
// state between steps:
//
//   y[b][t][c] = (residual ? x[b][t][c] : 0) + bias[c] + sum_{j < taps} w[c][j] * x[b][t - (taps-1) + j][c]      (then silu)
//
// w's last column weighs the current token.  Inputs before the step's first token come from state[b][taps-1][C] (fp32,
// oldest first); a sequence at position 0 has no past, whatever the state holds (a slot that another request used needs
// no clearing).  The input is a column slice of a wider matrix (a projection's output), any of the activation dtypes.
#include "common.cuh"

namespace llb {

constexpr int SC_THREADS = 128;
constexpr int SC_MAX_TAPS = 8;

// CPT neighbouring numbers of a row as fp32 (2: one 4-byte access in bf16, one 8-byte access in fp32).
template <typename T, int CPT>
__device__ __forceinline__ void sc_ld(const T* p, float (&o)[CPT]) {
  if constexpr (CPT == 1) o[0] = dt<T>::ld(p, 0);
  else if constexpr (sizeof(T) == 2) {
    const uint32_t u = *(const uint32_t*)p;
    o[0] = bf16_bits_to_f32(u & 0xffffu), o[1] = bf16_bits_to_f32(u >> 16);
  } else {
    const float2 u = *(const float2*)p;
    o[0] = u.x, o[1] = u.y;
  }
}
template <typename T, int CPT>
__device__ __forceinline__ void sc_st(T* p, const float (&v)[CPT]) {
  if constexpr (CPT == 1) dt<T>::st(p, 0, v[0]);
  else if constexpr (sizeof(T) == 2) *(uint32_t*)p = (uint32_t)f32_to_bf16_bits(v[0]) | ((uint32_t)f32_to_bf16_bits(v[1]) << 16);
  else *(float2*)p = make_float2(v[0], v[1]);
}

// grid (channel tiles, time tiles, B).  A thread owns CPT neighbouring channels and slides a window of TAPS inputs over its
// time tile.  fuse_state: the launch has ONE time tile and the thread also writes the new state (it has read the old one already).
template <typename TX, typename TY, int TAPS, int CPT>
__global__ void __launch_bounds__(SC_THREADS) short_conv_kernel(const TX* __restrict__ x, int x_stride, int col0,
                                                                const float* __restrict__ w, const float* __restrict__ bias,
                                                                float* __restrict__ state, const int32_t* __restrict__ pos_ids,
                                                                TY* __restrict__ y, int y_stride, int T, int C,
                                                                int t_tile, int residual, int act_silu, int fuse_state) {
  const int c = (blockIdx.x * SC_THREADS + threadIdx.x) * CPT;
  if (c >= C) return;
  const int b = blockIdx.z;
  const int t0 = blockIdx.y * t_tile, t1 = min(T, t0 + t_tile);
  const bool fresh = pos_ids[0] == 0;
  constexpr int HIST = TAPS - 1;
  float wr[TAPS][CPT], win[TAPS][CPT], bs[CPT];      // win[j] = input at time t - HIST + j (slot HIST: the current token)
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
#pragma unroll
    for (int e = 0; e < CPT; ++e) wr[j][e] = w[(size_t)(c + e) * TAPS + j];
#pragma unroll
  for (int e = 0; e < CPT; ++e) bs[e] = bias ? bias[c + e] : 0.f;
  const TX* xb = x + (size_t)b * T * x_stride + col0 + c;
  float* sb = state + (size_t)b * HIST * C + c;
#pragma unroll
  for (int j = 0; j < HIST; ++j) {
    const int s = t0 - HIST + j;
#pragma unroll
    for (int e = 0; e < CPT; ++e) win[j][e] = 0.f;
    if (s >= 0) sc_ld<TX, CPT>(xb + (size_t)s * x_stride, win[j]);
    else if (!fresh)
#pragma unroll
      for (int e = 0; e < CPT; ++e) win[j][e] = sb[(size_t)(HIST + s) * C + e];
  }
  auto token = [&](int t, const float (&cur)[CPT]) {
    float acc[CPT];
#pragma unroll
    for (int e = 0; e < CPT; ++e) {
      win[HIST][e] = cur[e];
      acc[e] = bs[e];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc[e] += wr[j][e] * win[j][e];
      if (residual) acc[e] += cur[e];
      if (act_silu) acc[e] = acc[e] / (1.f + expf(-acc[e]));
#pragma unroll
      for (int j = 0; j < HIST; ++j) win[j][e] = win[j + 1][e];
    }
    sc_st<TY, CPT>(y + ((size_t)b * T + t) * y_stride + c, acc);
  };
  int t = t0;
  for (; t + 8 <= t1; t += 8) {                      // the loads of eight tokens are in flight together
    float cur[8][CPT];
#pragma unroll
    for (int k = 0; k < 8; ++k) sc_ld<TX, CPT>(xb + (size_t)(t + k) * x_stride, cur[k]);
#pragma unroll
    for (int k = 0; k < 8; ++k) token(t + k, cur[k]);
  }
  for (; t < t1; ++t) {
    float cur[CPT];
    sc_ld<TX, CPT>(xb + (size_t)t * x_stride, cur);
    token(t, cur);
  }
  if (fuse_state) {
#pragma unroll
    for (int j = 0; j < HIST; ++j)
#pragma unroll
      for (int e = 0; e < CPT; ++e) sb[(size_t)j * C + e] = win[j][e];
  }
}

// The new state after a step of T tokens: the last taps-1 inputs (old state entries where the step is shorter).  One thread
// per (sequence, channel) reads everything it needs before it writes.
template <typename TX>
__global__ void short_conv_state_kernel(const TX* __restrict__ x, int x_stride, int col0, float* __restrict__ state,
                                        const int32_t* __restrict__ pos_ids, int T, int C, int taps) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int b = blockIdx.y;
  const bool fresh = pos_ids[0] == 0;
  const int hist = taps - 1;
  const TX* xb = x + (size_t)b * T * x_stride + col0 + c;
  float* sb = state + (size_t)b * hist * C + c;
  float nv[SC_MAX_TAPS - 1];
#pragma unroll
  for (int j = 0; j < SC_MAX_TAPS - 1; ++j) {
    float v = 0.f;
    if (j < hist) {
      const int s = T - hist + j;
      if (s >= 0) v = dt<TX>::ld(xb, (size_t)s * x_stride);
      else if (!fresh) v = sb[(size_t)(hist + s) * C];
    }
    nv[j] = v;
  }
#pragma unroll
  for (int j = 0; j < SC_MAX_TAPS - 1; ++j)
    if (j < hist) sb[(size_t)j * C] = nv[j];
}

template <typename TX, typename TY, int TAPS>
static int short_conv_launch(const void* x, int x_stride, int col0, const float* w, const float* bias, float* state,
                             const int32_t* pos_ids, void* y, int y_stride, int B, int T, int C, int flags, cudaStream_t st) {
  // pairs of channels where every row starts on a pair's boundary and the channels are many
  const bool pair = ((C | col0 | x_stride | y_stride) & 1) == 0 && ((uintptr_t)x & (2 * sizeof(TX) - 1)) == 0 &&
                    ((uintptr_t)y & (2 * sizeof(TY) - 1)) == 0 && C >= 2 * SC_THREADS;
  const int per = SC_THREADS * (pair ? 2 : 1);
  // time tiles: enough blocks to fill the device, at least 32 tokens each (every tile re-reads TAPS - 1 inputs)
  const int ctiles = (C + per - 1) / per;
  int tiles = max(1, min((T + 31) / 32, (16 * sm_count() + ctiles * B - 1) / (ctiles * B)));
  const int t_tile = ((T + tiles - 1) / tiles + 7) / 8 * 8;
  tiles = (T + t_tile - 1) / t_tile;
  const int fuse = tiles == 1 && state != nullptr;
  const dim3 grid(ctiles, tiles, B);
  if (pair)
    short_conv_kernel<TX, TY, TAPS, 2><<<grid, SC_THREADS, 0, st>>>((const TX*)x, x_stride, col0, w, bias, state, pos_ids, (TY*)y, y_stride,
                                                                    T, C, t_tile, flags & 1, (flags >> 1) & 1, fuse);
  else
    short_conv_kernel<TX, TY, TAPS, 1><<<grid, SC_THREADS, 0, st>>>((const TX*)x, x_stride, col0, w, bias, state, pos_ids, (TY*)y, y_stride,
                                                                    T, C, t_tile, flags & 1, (flags >> 1) & 1, fuse);
  LL_LAUNCH_OK("short_conv_kernel");
  if (!fuse && TAPS > 1) {
    short_conv_state_kernel<TX><<<dim3((C + 127) / 128, B), 128, 0, st>>>((const TX*)x, x_stride, col0, state, pos_ids, T, C, TAPS);
    LL_LAUNCH_OK("short_conv_state_kernel");
  }
  return LL_OK;
}

}  // namespace llb

using namespace llb;

extern "C" {

int ll_short_conv(const void* x, int x_dtype, int x_stride, int col0, const float* w, const float* bias, float* state,
                  const int32_t* pos_ids, void* y, int y_dtype, int y_stride, int B, int T, int C, int taps, int flags,
                  ll_stream stream) {
  LL_CHECK_ARG(x && w && state && pos_ids && y, "short_conv: null pointer");
  LL_CHECK_ARG(B >= 0 && T >= 0 && C > 0 && taps >= 1 && taps <= SC_MAX_TAPS && x_stride >= col0 + C && y_stride >= C,
               "bad short_conv arguments (taps up to %d)", SC_MAX_TAPS);
  if (B == 0 || T == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
#define LL_SC_T(TX, TY, TAPS) \
  case TAPS: return short_conv_launch<TX, TY, TAPS>(x, x_stride, col0, w, bias, state, pos_ids, y, y_stride, B, T, C, flags, st)
#define LL_SC(TX, TY)                                                                                     \
  switch (taps) {                                                                                         \
    LL_SC_T(TX, TY, 1); LL_SC_T(TX, TY, 2); LL_SC_T(TX, TY, 3); LL_SC_T(TX, TY, 4);                       \
    LL_SC_T(TX, TY, 5); LL_SC_T(TX, TY, 6); LL_SC_T(TX, TY, 7); LL_SC_T(TX, TY, 8);              \
  }
  if (x_dtype == LL_F32 && y_dtype == LL_F32) { LL_SC(float, float) }
  if (x_dtype == LL_F32 && y_dtype == LL_BF16) { LL_SC(float, __nv_bfloat16) }
  if (x_dtype == LL_BF16 && y_dtype == LL_BF16) { LL_SC(__nv_bfloat16, __nv_bfloat16) }
#undef LL_SC
#undef LL_SC_T
  set_error("short_conv: unsupported dtypes %d -> %d", x_dtype, y_dtype);
  return LL_ERR_UNSUPPORTED;
}

}  // extern "C"
