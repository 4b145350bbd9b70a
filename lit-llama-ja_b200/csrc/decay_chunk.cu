// The linear recurrence of decay_scan.cu for prompts in bf16, on tensor cores: with one decay per head and token (or one constant
// per head) the walk over tokens can be cut into chunks of 64 whose work is matrix products.  Per (sequence, head), G_t the sum of
// log a over the chunk up to token t:
//
//   collect   D_c = sum_s e^(G_last - G_s) (ks_s k_s) v_s^T             what a chunk adds to the state      (a block per chunk)
//   pass      S_c = e^(G_last) S_(c-1) + D_c                            the state before every chunk        (fp32, element by element)
//   read      y_t = qs ( sum_(s <= t) e^(G_t - G_s) ks_s (q_t.k_s) v_s + e^(G_t) S_(c-1)^T q_t ) + skip v_t     (a block per chunk)
//
// q, k and v are bf16 as they stand, so only the fp32 factors have to be split for the bf16 tensor cores (fp32 accumulation):
// e^(..) ks k enters D as three bf16 terms (24 bits: what is carried on is as exact as the walk's fp32), the chunk's weights and
// the state meet v and q as two terms (16 bits, the sum of both products in fp32).  Sums of log a are formed in fp64, so that the
// difference of two of them keeps its digits whatever lies before it in the chunk.  The state handed on is fp32.
#include "chunk_mma.cuh"

namespace llb {

// Blocks of eight warps: four rows of 16 x two halves of the block's PT value columns (64, or 128 for wide heads).  Everything a
// block reads is requested before anything is worked on, so that a block waits for memory about once.

// G[t] = sum over the chunk's tokens up to t of log a (tokens past the end: a = 1), by the first warp, two tokens a lane
__device__ __forceinline__ void dc_log_sums(const float* __restrict__ a, int a_row, int h, size_t m0, int len, double* G) {
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x;
  double v[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int t = 2 * lane + e;
    v[e] = t < len ? fmax((double)logf(a[(m0 + t) * a_row + h]), DC_LOG_MIN) : 0.0;
  }
  dc_running_sums(v, G);
}

// grid (chunks * p tiles, H, B): D_c into dst[((b * H + h) * chunks + c)][n][p], e^(G_last) into total[(b * H + h) * chunks + c].
// NP: n rounded up to 16, 32, 64 or 128.
template <int NP, int PT, bool SILU>
__global__ void __launch_bounds__(DC_THREADS, 2) decay_collect_kernel(const __nv_bfloat16* __restrict__ k, int k_stride,
                                                                      const __nv_bfloat16* __restrict__ v, int v_stride,
                                                                      const float* __restrict__ a, int a_row, const float* __restrict__ ks,
                                                                      float* __restrict__ dst, float* __restrict__ total, int Tn, int H,
                                                                      int qk_heads, int n, int p, int ptiles) {
  constexpr int LK = NP + 8, LV = PT + 8, NF = PT / 16;        // NF: 8-column fragments of a warp's half
  extern __shared__ __align__(16) unsigned char dc_smem[];
  __nv_bfloat16* Ks = (__nv_bfloat16*)dc_smem;                // [3 terms][64][LK]
  __nv_bfloat16* Vs = Ks + 3 * DC_L * LK;                     // [64][LV]
  __shared__ double G[DC_L];
  __shared__ float wgt[DC_L];
  const int c = blockIdx.x / ptiles, p0 = (blockIdx.x - c * ptiles) * PT, h = blockIdx.y, b = blockIdx.z, g = h / (H / qk_heads);
  const int chunks = gridDim.x / ptiles, t0 = c * DC_L, len = min(DC_L, Tn - t0), tid = threadIdx.x;
  const size_t m0 = (size_t)b * Tn + t0;
  DcTile<NP> kt;
  DcTile<PT> vt;
  kt.load(k + m0 * k_stride + (size_t)g * n, k_stride, len, n);
  vt.load(v + m0 * v_stride + (size_t)h * p + p0, v_stride, len, p - p0);
  const float ksv = (tid < len && ks) ? ks[(m0 + tid) * H + h] : 1.f;
  dc_log_sums(a, a_row, h, m0, len, G);
  vt.template store<SILU>(Vs, LV);
  __syncthreads();
  if (tid < DC_L) wgt[tid] = tid < len ? expf((float)(G[DC_L - 1] - G[tid])) * ksv : 0.f;
  if (tid == 0 && p0 == 0) total[((size_t)b * H + h) * chunks + c] = expf((float)G[DC_L - 1]);
  __syncthreads();
#pragma unroll
  for (int it = 0; it < DcTile<NP>::IT; ++it) {
    const int i = it * DC_THREADS + tid, s = i / (NP / 8), ch = (i % (NP / 8)) * 8;
    if (i >= DcTile<NP>::UNITS) break;
    const uint4 u = dc_in8<SILU>(kt.u[it]);
    const float w = wgt[s];
    const uint32_t in[4] = {u.x, u.y, u.z, u.w};
    uint32_t out[3][4];
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      float x0 = bf16_bits_to_f32(in[q] & 0xffffu) * w, x1 = bf16_bits_to_f32(in[q] >> 16) * w;
      out[0][q] = dc_term(x0, x1);
      out[1][q] = dc_term(x0, x1);
      out[2][q] = pack_bf16(x0, x1);
    }
#pragma unroll
    for (int z = 0; z < 3; ++z) *(uint4*)&Ks[(z * DC_L + s) * LK + ch] = make_uint4(out[z][0], out[z][1], out[z][2], out[z][3]);
  }
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31, c0 = (warp >> 2) * (PT / 2);
  float* D = dst + (((size_t)b * H + h) * chunks + c) * (size_t)n * p;
#pragma unroll 1
  for (int mt = warp & 3; mt < NP / 16; mt += 4) {
    if (mt * 16 >= n) break;
    float acc[NF][4];
#pragma unroll
    for (int f = 0; f < NF; ++f) acc[f][0] = acc[f][1] = acc[f][2] = acc[f][3] = 0.f;
#pragma unroll
    for (int st = 0; st < DC_L / 16; ++st) {
      uint32_t bf[NF / 2][4];
#pragma unroll
      for (int d = 0; d < NF / 2; ++d)
        dc_ldmatrix_trans(bf[d], &Vs[(st * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LV + c0 + d * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int z = 2; z >= 0; --z) {                          // the smallest term first
        uint32_t af[4];
        dc_ldmatrix_trans(af, &Ks[(z * DC_L + st * 16 + (lane & 7) + (lane >> 4) * 8) * LK + mt * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
        for (int d = 0; d < NF / 2; ++d) {
          mma_bf16_16816(acc[2 * d], af[0], af[1], af[2], af[3], bf[d][0], bf[d][1]);
          mma_bf16_16816(acc[2 * d + 1], af[0], af[1], af[2], af[3], bf[d][2], bf[d][3]);
        }
      }
    }
#pragma unroll
    for (int f = 0; f < NF; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = mt * 16 + (lane >> 2) + e * 8, col = p0 + c0 + f * 8 + (lane & 3) * 2;
        if (i < n && col < p) *(float2*)(D + (size_t)i * p + col) = make_float2(acc[f][2 * e], acc[f][2 * e + 1]);
      }
  }
}

// Per (sequence, head), two neighbouring elements of the state a thread: D_c is replaced by the state before chunk c, the state
// after the last chunk goes back to `state`.
__global__ void __launch_bounds__(128) decay_pass_kernel(float* __restrict__ chunk_state, const float* __restrict__ total,
                                                         float* __restrict__ state, const int32_t* __restrict__ pos_ids, int chunks,
                                                         int np2) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= np2) return;
  const size_t bh = blockIdx.y;
  float2* D = (float2*)chunk_state + bh * chunks * np2 + i;
  float2* S = (float2*)state + bh * np2 + i;
  const float* tot = total + bh * chunks;
  float2 s = pos_ids[0] == 0 ? make_float2(0.f, 0.f) : *S;
  constexpr int AHEAD = 16;                                   // chunks whose loads are in flight together
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
    float2 d[AHEAD];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) d[j] = c0 + j < chunks ? D[(size_t)(c0 + j) * np2] : make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
      if (c0 + j < chunks) {
        const float w = tot[c0 + j];
        D[(size_t)(c0 + j) * np2] = s;
        s = make_float2(w * s.x + d[j].x, w * s.y + d[j].y);
      }
  }
  *S = s;
}

// grid (chunks * p tiles, H, B).  A warp owns 16 consecutive tokens and half of the block's columns; its queries come from global
// memory straight into fragments.
template <int NP, int PT, bool SILU>
__global__ void __launch_bounds__(DC_THREADS, 2) decay_read_kernel(
    const __nv_bfloat16* __restrict__ q, int q_stride, const __nv_bfloat16* __restrict__ k, int k_stride, const __nv_bfloat16* __restrict__ v,
    int v_stride, const float* __restrict__ a, int a_row, const float* __restrict__ ks, const float* __restrict__ skip, float qs,
    const float* __restrict__ chunk_state, const int32_t* __restrict__ pos_ids, float* __restrict__ y, int Tn, int H, int qk_heads, int n,
    int p, int ptiles) {
  constexpr int LK = NP + 8, LV = PT + 8, NF = PT / 16;
  extern __shared__ __align__(16) unsigned char dc_smem[];
  __nv_bfloat16* Ks = (__nv_bfloat16*)dc_smem;                // [64][LK]
  __nv_bfloat16* Vs = Ks + DC_L * LK;                         // [64][LV]
  __nv_bfloat16* Ss = Vs + DC_L * LV;                         // [2 terms][NP][LV]
  __shared__ double G[DC_L];
  __shared__ float kw[DC_L];
  const int c = blockIdx.x / ptiles, p0 = (blockIdx.x - c * ptiles) * PT, h = blockIdx.y, b = blockIdx.z, g = h / (H / qk_heads);
  const int chunks = gridDim.x / ptiles, t0 = c * DC_L, len = min(DC_L, Tn - t0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, row0 = (warp & 3) * 16, c0 = (warp >> 2) * (PT / 2);
  const size_t m0 = (size_t)b * Tn + t0;
  const bool has_state = c > 0 || pos_ids[0] != 0;
  const float* S = chunk_state + (((size_t)b * H + h) * chunks + c) * (size_t)n * p;
  DcTile<NP> kt;
  DcTile<PT> vt;
  kt.load(k + m0 * k_stride + (size_t)g * n, k_stride, len, n);
  vt.load(v + m0 * v_stride + (size_t)h * p + p0, v_stride, len, p - p0);
  const float ksv = (tid < len && ks) ? ks[(m0 + tid) * H + h] : 1.f;
  // the state's rows in rounds of eight 16-byte units per thread: the first round is requested with the keys and values
  constexpr int SU = NP * (PT / 4), SR = (SU + 8 * DC_THREADS - 1) / (8 * DC_THREADS);
  float4 sv[8];
  auto state_load = [&](int rd) {
#pragma unroll
    for (int it = 0; it < 8; ++it) {
      const int i = (rd * 8 + it) * DC_THREADS + tid, r = i / (PT / 4), col = (i % (PT / 4)) * 4;
      sv[it] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < SU && r < n && p0 + col < p) sv[it] = *(const float4*)(S + (size_t)r * p + p0 + col);
    }
  };
  if (has_state) state_load(0);
  kt.template store<SILU>(Ks, LK);
  vt.template store<SILU>(Vs, LV);
  if (has_state) {
#pragma unroll
    for (int rd = 0; rd < SR; ++rd) {
#pragma unroll
      for (int it = 0; it < 8; ++it) {
        const int i = (rd * 8 + it) * DC_THREADS + tid, r = i / (PT / 4), col = (i % (PT / 4)) * 4;
        if (i >= SU) break;
        float4 f = sv[it];
        const uint32_t h0 = dc_term(f.x, f.y), h1 = dc_term(f.z, f.w);
        *(uint2*)&Ss[r * LV + col] = make_uint2(h0, h1);
        *(uint2*)&Ss[(NP + r) * LV + col] = make_uint2(pack_bf16(f.x, f.y), pack_bf16(f.z, f.w));
      }
      if (rd + 1 < SR) state_load(rd + 1);
    }
  }
  if (tid < DC_L) kw[tid] = tid < len ? ksv * qs : 0.f;
  dc_log_sums(a, a_row, h, m0, len, G);
  // query fragments: rows (lane / 4) and + 8 of the warp's 16, columns (lane % 4) * 2 and + 8 of every 16
  uint32_t qf[NP / 16][4];
  const int r0 = row0 + (lane >> 2);
#pragma unroll
  for (int kk = 0; kk < NP / 16; ++kk)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = r0 + (e & 1) * 8, col = kk * 16 + (lane & 3) * 2 + (e >> 1) * 8;
      qf[kk][e] = (r < len && col < n) ? dc_in2<SILU>(*(const uint32_t*)(q + (m0 + r) * q_stride + (size_t)g * n + col)) : 0u;
    }
  __syncthreads();
  if (row0 >= len) return;
  float o[NF][4];
#pragma unroll
  for (int f = 0; f < NF; ++f) o[f][0] = o[f][1] = o[f][2] = o[f][3] = 0.f;
  const double g0 = G[r0], g1 = G[r0 + 8];
  if (has_state) {
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk)
#pragma unroll
      for (int z = 1; z >= 0; --z)
#pragma unroll
        for (int d = 0; d < NF / 2; ++d) {
          uint32_t bf[4];
          dc_ldmatrix_trans(bf, &Ss[(z * NP + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LV + c0 + d * 16 + (lane >> 4) * 8]);
          mma_bf16_16816(o[2 * d], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], bf[0], bf[1]);
          mma_bf16_16816(o[2 * d + 1], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], bf[2], bf[3]);
        }
    const float e0 = expf((float)g0) * qs, e1 = expf((float)g1) * qs;
#pragma unroll
    for (int f = 0; f < NF; ++f) o[f][0] *= e0, o[f][1] *= e0, o[f][2] *= e1, o[f][3] *= e1;
  }
#pragma unroll
  for (int st = 0; st < DC_L / 16; ++st) {                    // 16 keys at a time, none that lie after all of the warp's tokens
    if (st * 16 > row0) break;
    float sc[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk) {
      uint32_t bf[4];
      dc_ldmatrix(bf, &Ks[(st * 16 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8]);
      mma_bf16_16816(sc[0], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], bf[0], bf[1]);
      mma_bf16_16816(sc[1], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], bf[2], bf[3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int s = st * 16 + j * 8 + (lane & 3) * 2 + (e & 1), r = r0 + (e >> 1) * 8;
        sc[j][e] = s <= r ? sc[j][e] * (expf((float)((e >> 1 ? g1 : g0) - G[s])) * kw[s]) : 0.f;
      }
    uint32_t ah[4], al[4];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      ah[2 * j] = dc_term(sc[j][0], sc[j][1]), al[2 * j] = pack_bf16(sc[j][0], sc[j][1]);
      ah[2 * j + 1] = dc_term(sc[j][2], sc[j][3]), al[2 * j + 1] = pack_bf16(sc[j][2], sc[j][3]);
    }
#pragma unroll
    for (int d = 0; d < NF / 2; ++d) {
      uint32_t bf[4];
      dc_ldmatrix_trans(bf, &Vs[(st * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LV + c0 + d * 16 + (lane >> 4) * 8]);
      mma_bf16_16816(o[2 * d], al[0], al[1], al[2], al[3], bf[0], bf[1]);
      mma_bf16_16816(o[2 * d + 1], al[0], al[1], al[2], al[3], bf[2], bf[3]);
      mma_bf16_16816(o[2 * d], ah[0], ah[1], ah[2], ah[3], bf[0], bf[1]);
      mma_bf16_16816(o[2 * d + 1], ah[0], ah[1], ah[2], ah[3], bf[2], bf[3]);
    }
  }
  const float sk = skip ? skip[h] : 0.f;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = r0 + e * 8;
    if (r >= len) continue;
    float* yr = y + (m0 + r) * (size_t)H * p + (size_t)h * p + p0 + c0;
#pragma unroll
    for (int f = 0; f < NF; ++f) {
      const int col = f * 8 + (lane & 3) * 2;
      if (p0 + c0 + col >= p) continue;
      float v0 = o[f][2 * e], v1 = o[f][2 * e + 1];
      if (skip) {
        v0 += sk * __bfloat162float(Vs[r * LV + c0 + col]);
        v1 += sk * __bfloat162float(Vs[r * LV + c0 + col + 1]);
      }
      *(float2*)(yr + col) = make_float2(v0, v1);
    }
  }
}

template <int NP, int PT, bool SILU>
static int decay_chunked_launch(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const float* a,
                                int a_row, const float* ks, const float* skip, float qs, float* state, const int32_t* pos_ids, float* y,
                                int B, int Tn, int H, int qk_heads, int n, int p, float* scratch, cudaStream_t st) {
  const int chunks = (Tn + DC_L - 1) / DC_L, ptiles = (p + PT - 1) / PT, np2 = n * p / 2;
  float* chunk_state = scratch;
  float* total = scratch + (size_t)B * H * chunks * n * p;
  const dim3 grid(chunks * ptiles, H, B);
  constexpr int smem_c = (3 * DC_L * (NP + 8) + DC_L * (PT + 8)) * 2, smem_r = (DC_L * (NP + 8) + DC_L * (PT + 8) + 2 * NP * (PT + 8)) * 2;
  static bool sized = false;
  if (!sized) {
    LL_CUDA(cudaFuncSetAttribute(decay_collect_kernel<NP, PT, SILU>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_c));
    LL_CUDA(cudaFuncSetAttribute(decay_read_kernel<NP, PT, SILU>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_r));
    sized = true;
  }
  typedef const __nv_bfloat16* in_t;
  decay_collect_kernel<NP, PT, SILU><<<grid, DC_THREADS, smem_c, st>>>((in_t)k, k_stride, (in_t)v, v_stride, a, a_row, ks, chunk_state, total, Tn, H,
                                                                  qk_heads, n, p, ptiles);
  LL_LAUNCH_OK("decay_collect_kernel");
  decay_pass_kernel<<<dim3((np2 + 127) / 128, B * H), 128, 0, st>>>(chunk_state, total, state, pos_ids, chunks, np2);
  LL_LAUNCH_OK("decay_pass_kernel");
  decay_read_kernel<NP, PT, SILU><<<grid, DC_THREADS, smem_r, st>>>((in_t)q, q_stride, (in_t)k, k_stride, (in_t)v, v_stride, a, a_row, ks, skip, qs,
                                                               chunk_state, pos_ids, y, Tn, H, qk_heads, n, p, ptiles);
  LL_LAUNCH_OK("decay_read_kernel");
  return LL_OK;
}

}  // namespace llb

using namespace llb;

extern "C" {

int ll_decay_chunked_supported(int dtype, int T, int n, int p, int q_stride, int k_stride, int v_stride) {
  return dtype == LL_BF16 && T >= DC_L && n % 8 == 0 && n <= 128 && p % 8 == 0 && ((q_stride | k_stride | v_stride) & 7) == 0;
}

size_t ll_decay_chunked_scratch_bytes(int B, int T, int H, int n, int p) {
  const size_t chunks = (T + DC_L - 1) / DC_L;
  return (size_t)B * H * chunks * ((size_t)n * p + 1) * sizeof(float);
}

int ll_decay_chunked(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, int dtype, const float* a,
                     int a_constant, int act_silu, const float* ks, const float* skip, float qs, float* state, const int32_t* pos_ids,
                     float* y, int B, int T, int H, int qk_heads, int n, int p, float* scratch, ll_stream stream) {
  LL_CHECK_ARG(q && k && v && a && state && pos_ids && y && scratch, "decay_chunked: null pointer");
  LL_CHECK_ARG(B >= 0 && T >= 0 && H > 0 && qk_heads > 0 && H % qk_heads == 0 && n > 0 && p > 0, "bad decay_chunked arguments");
  if (B == 0 || T == 0) return LL_OK;
  const uintptr_t at = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)y | (uintptr_t)scratch;
  if (!ll_decay_chunked_supported(dtype, T, n, p, q_stride, k_stride, v_stride) || (at & 15) != 0 || (long long)B * H > 65535) {
    set_error("decay_chunked: bf16, at least %d tokens, n and p in multiples of 8 (n up to 128), rows on 16-byte boundaries", DC_L);
    return LL_ERR_UNSUPPORTED;
  }
  cudaStream_t st = (cudaStream_t)stream;
  const int a_row = a_constant ? 0 : H;
#define LL_DC_S(NP, SILU)                                                                                                              \
  return p <= 64 ? decay_chunked_launch<NP, 64, SILU>(q, q_stride, k, k_stride, v, v_stride, a, a_row, ks, skip, qs, state, pos_ids, y, B, T, \
                                                      H, qk_heads, n, p, scratch, st)                                                        \
                 : decay_chunked_launch<NP, 128, SILU>(q, q_stride, k, k_stride, v, v_stride, a, a_row, ks, skip, qs, state, pos_ids, y, B, T, \
                                                       H, qk_heads, n, p, scratch, st)
#define LL_DC(NP)                  \
  if (n <= NP) {                   \
    if (act_silu) LL_DC_S(NP, true); \
    LL_DC_S(NP, false);            \
  }
  LL_DC(16) LL_DC(32) LL_DC(64) LL_DC(128)
#undef LL_DC
#undef LL_DC_S
  return LL_ERR_UNSUPPORTED;
}

}  // extern "C"
