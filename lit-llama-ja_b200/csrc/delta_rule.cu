// Gated delta rule, token by token.  Per sequence b and head h, with S an n x p matrix and q, k of head h / (H / qk_heads):
//
//   k^ = k / sqrt(|k|^2 + e),   q^ = q / sqrt(|q|^2 + e) * qs,   g = exp(-exp(a_log) softplus(raw_a + dt_bias)),   beta = sigmoid(raw_b)
//   S <- g S;      u = beta (v - S^T k^);      S <- S + k^ u^T;      y = S^T q^
//
// q, k (raw: the short convolution's output), v and the two gate projections are column slices of matrices in the activation
// dtype; everything else, the state included, is fp32.  The state is carried in state[B][H][n][p]; a sequence at position 0 starts
// from zero whatever it holds.
//
// The walk reads what the memory returns for k and for q from the state BEFORE the token, in one sweep whose two sums are reduced
// together, so that a token costs one round of shuffles:  with w = beta (v - g k^.S) / |k|,
//   S'[i] = g S[i] + k[i] w,        y = qs / |q| * (g q.S + (q.k) w).
// The norms, q.k and the gates of a staged round are formed from the staged numbers, a warp per token.
#include "delta.cuh"

namespace llb {

constexpr int DR_THREADS = 128;
__host__ __device__ constexpr int dr_tokens(int npad) { return npad <= 64 ? 16 : npad <= 128 ? 8 : npad <= 256 ? 4 : 2; }

// grid (p tiles, H, B).  NP threads (consecutive lanes) share one column and split the n rows, NL rows each in registers,
// interleaved in quads (row(i) = ((i / 4) * NP + part) * 4 + i % 4: the lanes of a column read consecutive 16-byte units).
template <typename T, int NP, int NL>
__global__ void __launch_bounds__(DR_THREADS) delta_scan_kernel(
    const T* __restrict__ q, int q_stride, const T* __restrict__ k, int k_stride, const T* __restrict__ v, int v_stride,
    const T* __restrict__ raw_a, const T* __restrict__ raw_b, int gate_stride, const float* __restrict__ dt_bias,
    const float* __restrict__ a_log, float unit_eps, float qs, float* __restrict__ state, const int32_t* __restrict__ pos_ids,
    float* __restrict__ y, int Tn, int H, int qk_heads, int n, int p) {
  constexpr int PT = DR_THREADS / NP, NPAD = NP * NL, TC = dr_tokens(NPAD);
  __shared__ __align__(16) float s_k[TC][NPAD], s_q[TC][NPAD];
  __shared__ float s_v[TC][PT];
  __shared__ float s_g[TC], s_beta[TC], s_rk[TC], s_rq[TC], s_qk[TC];
  const int h = blockIdx.y, b = blockIdx.z, g = h / (H / qk_heads);
  const int part = threadIdx.x % NP, pl = threadIdx.x / NP, c = blockIdx.x * PT + pl;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool live = c < p;
#define DR_ROW(i) ((((i) >> 2) * NP + part) * 4 + ((i) & 3))
  float S[NL];
  float* sp = state + (((size_t)b * H + h) * n) * p;
  const bool fresh = pos_ids[0] == 0;
#pragma unroll
  for (int i = 0; i < NL; ++i) S[i] = (!fresh && live && DR_ROW(i) < n) ? sp[(size_t)DR_ROW(i) * p + c] : 0.f;
  const float dtb = dt_bias[h], al = a_log[h];
  // the next round's tokens are fetched (raw) into registers while this round's are consumed from shared memory
  constexpr int IT = TC * NPAD / DR_THREADS, VIT = (TC * PT + DR_THREADS - 1) / DR_THREADS;
  T rk[IT], rq[IT], rv[VIT], ra, rb;
  auto fetch = [&](int t0) {
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int idx = it * DR_THREADS + threadIdx.x, tt = idx / NPAD, i = idx - tt * NPAD;
      const size_t m = (size_t)b * Tn + t0 + tt;
      const bool ok = t0 + tt < Tn && i < n;
      rk[it] = k[ok ? m * k_stride + (size_t)g * n + i : 0];
      rq[it] = q[ok ? m * q_stride + (size_t)g * n + i : 0];
    }
#pragma unroll
    for (int it = 0; it < VIT; ++it) {
      const int idx = it * DR_THREADS + threadIdx.x, tt = idx / PT, col = blockIdx.x * PT + idx - tt * PT;
      const bool ok = tt < TC && t0 + tt < Tn && col < p;
      rv[it] = v[ok ? ((size_t)b * Tn + t0 + tt) * v_stride + (size_t)h * p + col : 0];
    }
    const bool ok = threadIdx.x < TC && t0 + (int)threadIdx.x < Tn;
    const size_t at = ok ? ((size_t)b * Tn + t0 + threadIdx.x) * gate_stride + h : 0;
    ra = raw_a[at], rb = raw_b[at];
  };
  fetch(0);
  for (int t0 = 0; t0 < Tn; t0 += TC) {
    const int nt = min(TC, Tn - t0);
    __syncthreads();
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int idx = it * DR_THREADS + threadIdx.x, tt = idx / NPAD, i = idx - tt * NPAD;
      const bool ok = t0 + tt < Tn && i < n;
      s_k[tt][i] = ok ? dt<T>::ld(&rk[it], 0) : 0.f;
      s_q[tt][i] = ok ? dt<T>::ld(&rq[it], 0) : 0.f;
    }
#pragma unroll
    for (int it = 0; it < VIT; ++it) {
      const int idx = it * DR_THREADS + threadIdx.x, tt = idx / PT, cc = idx - tt * PT;
      if (tt < TC) s_v[tt][cc] = (t0 + tt < Tn && blockIdx.x * PT + cc < p) ? dt<T>::ld(&rv[it], 0) : 0.f;
    }
    if (threadIdx.x < TC) {
      s_g[threadIdx.x] = expf(delta_log_decay(dt<T>::ld(&ra, 0), dtb, al));
      s_beta[threadIdx.x] = delta_strength(dt<T>::ld(&rb, 0));
    }
    __syncthreads();
    if (t0 + TC < Tn) fetch(t0 + TC);
    for (int tt = warp; tt < nt; tt += DR_THREADS / 32) {
      float kk = 0.f, qq = 0.f, qk = 0.f;
      for (int i = lane; i < NPAD; i += 32) {
        const float kv = s_k[tt][i], qv = s_q[tt][i];
        kk += kv * kv, qq += qv * qv, qk += qv * kv;
      }
      kk = warp_sum(kk), qq = warp_sum(qq), qk = warp_sum(qk);
      if (lane == 0) s_rk[tt] = 1.f / sqrtf(kk + unit_eps), s_rq[tt] = qs / sqrtf(qq + unit_eps), s_qk[tt] = qk;
    }
    __syncthreads();
    for (int tt = 0; tt < nt; ++tt) {
      float ck[4] = {0.f, 0.f, 0.f, 0.f}, cq[4] = {0.f, 0.f, 0.f, 0.f};
      float4 k4[NL / 4];
#pragma unroll
      for (int i4 = 0; i4 < NL; i4 += 4) {
        const int at = ((i4 >> 2) * NP + part) * 4;
        k4[i4 >> 2] = *(const float4*)&s_k[tt][at];
        const float4 kv = k4[i4 >> 2], qv = *(const float4*)&s_q[tt][at];
        ck[0] += kv.x * S[i4], ck[1] += kv.y * S[i4 + 1], ck[2] += kv.z * S[i4 + 2], ck[3] += kv.w * S[i4 + 3];
        cq[0] += qv.x * S[i4], cq[1] += qv.y * S[i4 + 1], cq[2] += qv.z * S[i4 + 2], cq[3] += qv.w * S[i4 + 3];
      }
      float sk = (ck[0] + ck[1]) + (ck[2] + ck[3]), sq = (cq[0] + cq[1]) + (cq[2] + cq[3]);
#pragma unroll
      for (int o = NP / 2; o > 0; o >>= 1) {
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
      }
      const float gt = s_g[tt], rkt = s_rk[tt];
      const float w = rkt * (s_beta[tt] * (s_v[tt][pl] - gt * rkt * sk));
#pragma unroll
      for (int i4 = 0; i4 < NL; i4 += 4) {
        const float4 kv = k4[i4 >> 2];
        S[i4] = gt * S[i4] + kv.x * w, S[i4 + 1] = gt * S[i4 + 1] + kv.y * w;
        S[i4 + 2] = gt * S[i4 + 2] + kv.z * w, S[i4 + 3] = gt * S[i4 + 3] + kv.w * w;
      }
      if (part == 0 && live) y[((size_t)b * Tn + t0 + tt) * ((size_t)H * p) + (size_t)h * p + c] = s_rq[tt] * (gt * sq + s_qk[tt] * w);
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < NL; ++i)
      if (DR_ROW(i) < n) sp[(size_t)DR_ROW(i) * p + c] = S[i];
  }
#undef DR_ROW
}

struct DeltaArgs {
  const void *q, *k, *v, *raw_a, *raw_b;
  int q_stride, k_stride, v_stride, gate_stride;
  const float *dt_bias, *a_log;
  float unit_eps, qs;
  float* state;
  const int32_t* pos_ids;
  float* y;
  int B, T, H, qk_heads, n, p;
};

template <typename T, int NP, int NL>
static int delta_scan_launch(const DeltaArgs& A, cudaStream_t st) {
  constexpr int PT = DR_THREADS / NP;
  delta_scan_kernel<T, NP, NL><<<dim3((A.p + PT - 1) / PT, A.H, A.B), DR_THREADS, 0, st>>>(
      (const T*)A.q, A.q_stride, (const T*)A.k, A.k_stride, (const T*)A.v, A.v_stride, (const T*)A.raw_a, (const T*)A.raw_b, A.gate_stride,
      A.dt_bias, A.a_log, A.unit_eps, A.qs, A.state, A.pos_ids, A.y, A.T, A.H, A.qk_heads, A.n, A.p);
  LL_LAUNCH_OK("delta_scan_kernel");
  return LL_OK;
}

template <typename T>
static int delta_scan_dispatch(const DeltaArgs& A, cudaStream_t st) {
  // 16 rows per thread when that already gives half of the SMs a block, 8 when the heads are few (as in decay_scan.cu)
  int np16 = 1;
  while (np16 * 16 < A.n) np16 *= 2;
  const long long blocks16 = (long long)A.B * A.H * ((A.p + DR_THREADS / np16 - 1) / (DR_THREADS / np16));
  const int nl = (A.n > 256 || 2 * blocks16 >= sm_count()) ? 16 : 8;
  int np = 1;
  while (np * nl < A.n) np *= 2;
#define LL_DR(NP) return nl == 8 ? delta_scan_launch<T, NP, 8>(A, st) : delta_scan_launch<T, NP, 16>(A, st)
  switch (np) {
    case 1: LL_DR(1);
    case 2: LL_DR(2);
    case 4: LL_DR(4);
    case 8: LL_DR(8);
    case 16: LL_DR(16);
    default: LL_DR(32);
  }
#undef LL_DR
}

}  // namespace llb

using namespace llb;

extern "C" {

int ll_delta_scan(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const void* raw_a,
                  const void* raw_b, int gate_stride, int dtype, const float* dt_bias, const float* a_log, float unit_eps, float qs,
                  float* state, const int32_t* pos_ids, float* y, int B, int T, int H, int qk_heads, int n, int p, ll_stream stream) {
  LL_CHECK_ARG(q && k && v && raw_a && raw_b && dt_bias && a_log && state && pos_ids && y, "delta_scan: null pointer");
  LL_CHECK_ARG(B >= 0 && T >= 0 && H > 0 && qk_heads > 0 && H % qk_heads == 0 && n > 0 && p > 0 && gate_stride >= H,
               "bad delta_scan arguments");
  if (n > 32 * 16 || B > 65535 || H > 65535) {
    set_error("delta_scan: %d state rows per head (up to %d)", n, 32 * 16);
    return LL_ERR_UNSUPPORTED;
  }
  if (B == 0 || T == 0) return LL_OK;
  const DeltaArgs A{q, k, v, raw_a, raw_b, q_stride, k_stride, v_stride, gate_stride, dt_bias, a_log, unit_eps, qs, state, pos_ids, y,
                    B, T, H, qk_heads, n, p};
  if (dtype == LL_F32) return delta_scan_dispatch<float>(A, (cudaStream_t)stream);
  if (dtype == LL_BF16) return delta_scan_dispatch<__nv_bfloat16>(A, (cudaStream_t)stream);
  set_error("delta_scan: unsupported dtype %d", dtype);
  return LL_ERR_UNSUPPORTED;
}

}  // extern "C"
