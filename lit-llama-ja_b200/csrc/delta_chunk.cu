// The gated delta rule of delta_rule.cu for prompts in bf16, on tensor cores.  Within a chunk of 64 tokens, S_0 the state before it,
// G_t the sum of the log decays up to token t, k^_t = r_t k_t the unit keys and b_t the write strengths, what token t writes is
//
//   u_t = b_t (v_t - e^(G_t) S_0^T k^_t - sum_(s < t) e^(G_t - G_s) (k^_s.k^_t) u_s),       S_t = e^(G_t) S_0 + sum_(s <= t) e^(G_t - G_s) k^_s u_s^T
//
// a triangular system (I + L) U = diag(b) (V - diag(e^G) K^ S_0) whose matrix does not depend on the state:
//
//   prepare   X = (I + L)^-1;   W = X diag(b e^G) K^,   U_0 = X diag(b) V,   A_ts = e^(G_t - G_s) q^_t.k^_s (s <= t)   (a block per chunk)
//   pass      U = U_0 - W S_c;   S_(c+1) = e^(G_last) S_c + sum_s e^(G_last - G_s) k^_s u_s^T       (a block per column tile of a head,
//             which walks the chunks with its slice of the state in registers)
//   read      y_t = q^_t.( e^(G_t) S_c ) + sum_(s <= t) A_ts u_s                                  (a block per chunk and 64 columns)
//
// X is formed by substitution (8 x 8 blocks, then merged by halves), which holds for any keys: a series in powers of L would not.
// k, q and v are bf16 as they stand; the fp32 factors are split into bf16 terms (fp32 accumulation): three (24 bits) where X meets K
// and V - its rows cancel when keys repeat, and many small u add up in a read-out - and where U enters the state; two (16 bits, the
// three largest of the four products) where W meets the state and where A and the queries meet U and the state.
// Sums of log decays are fp64.  The state handed on is fp32.
#include "chunk_mma.cuh"
#include "delta.cuh"

namespace llb {

constexpr int DX_LD = DC_L + 4;                              // row pitch of the fp32 triangle
constexpr int DX_TMP = 36;

// Per (sequence, head, chunk) j, all of it written by `prepare` except what `pass` leaves for `read`:
struct DeltaScratch {
  float* fac;               // [64] e^(G_last - G_t) / |k_t|
  float* row;               // [64] e^(G_t) qs / |q_t|
  float* tot;               // e^(G_last)                                        (four floats apart)
  float* U0;                // [64][p]
  __nv_bfloat16* A;         // [2 terms][64][64]; only 16 x 16 blocks up to the diagonal are written
  __nv_bfloat16* U;         // [2 terms][64][p]                                  (pass)
  __nv_bfloat16* S;         // [2 terms][n][p], the state before the chunk       (pass)
  __nv_bfloat16* WK;        // [3][64][NP + 8]: two terms of W, then K, zeros beside n: an image of the stage in shared memory
};

struct DeltaChunkArgs {
  const __nv_bfloat16 *q, *k, *v, *raw_a, *raw_b;
  int q_stride, k_stride, v_stride, gate_stride;
  const float *dt_bias, *a_log;
  float unit_eps, qs;
  float* state;
  const int32_t* pos_ids;
  float* y;
  int T, H, qk_heads, n, p, chunks;
  DeltaScratch sc;
};

// four neighbouring numbers: o += a * x
__device__ __forceinline__ void fma4(float4& o, float a, const float4 x) {
  o.x = fmaf(a, x.x, o.x), o.y = fmaf(a, x.y, o.y), o.z = fmaf(a, x.z, o.z), o.w = fmaf(a, x.w, o.w);
}

// The inverse of a unit lower triangle in place, merged by halves: the block [r0 .. r0 + N)[c0 .. c0 + N), c0 = r0 - N, becomes
// -X_22 (L_21 X_11).  `pairs` merges side by side, a thread per four columns of a row (N * N / 4 threads a merge); two barriers.
template <int N>
__device__ __forceinline__ void dx_merge(float* X, float* tmp, int pairs) {
  constexpr int TPM = N * N / 4;
  const int z = threadIdx.x / TPM, e = threadIdx.x - z * TPM, i = e / (N / 4), j = (e % (N / 4)) * 4;
  const int r0 = (2 * z + 1) * N, c0 = 2 * z * N;
  float* tm = tmp + z * N * DX_TMP;
  if (z < pairs) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int k = 0; k < N; ++k) fma4(o, X[(r0 + i) * DX_LD + c0 + k], *(const float4*)&X[(c0 + k) * DX_LD + c0 + j]);
    *(float4*)&tm[i * DX_TMP + j] = o;
  }
  __syncthreads();
  if (z < pairs) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int k = 0; k < N; ++k) fma4(o, -X[(r0 + i) * DX_LD + r0 + k], *(const float4*)&tm[k * DX_TMP + j]);
    *(float4*)&X[(r0 + i) * DX_LD + c0 + j] = o;
  }
  __syncthreads();
}

// The same on tensor cores for N = 16, 32, a warp per 16 x 8 tile: both factors as three bf16 terms, the six largest products (24 bits).
template <int N>
__device__ __forceinline__ void dx_tile_product(const float* __restrict__ a, int lda, const float* __restrict__ b, int ldb, float (&acc)[4]) {
  const int lane = threadIdx.x & 31;
  acc[0] = acc[1] = acc[2] = acc[3] = 0.f;
#pragma unroll
  for (int kt = 0; kt < N / 16; ++kt) {
    uint32_t af[3][4], bf[3][2], t[3];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 x = *(const float2*)&a[((lane >> 2) + (e & 1) * 8) * lda + kt * 16 + (lane & 3) * 2 + (e >> 1) * 8];
      dc_terms<3>(x.x, x.y, t);
      af[0][e] = t[0], af[1][e] = t[1], af[2][e] = t[2];
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float* at = &b[(kt * 16 + (lane & 3) * 2 + e * 8) * ldb + (lane >> 2)];
      dc_terms<3>(at[0], at[ldb], t);
      bf[0][e] = t[0], bf[1][e] = t[1], bf[2][e] = t[2];
    }
#pragma unroll
    for (int sum = 2; sum >= 0; --sum)                        // the smallest products first
#pragma unroll
      for (int z = 0; z <= sum; ++z) dc_mma(acc, af[z], bf[sum - z][0], bf[sum - z][1]);
  }
}

template <int N>
__device__ __forceinline__ void dx_merge_mma(float* X, float* tmp, int pairs) {
  constexpr int MT = N / 16, TILES = MT * (N / 8);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int z = warp / TILES, e = warp - z * TILES, m = (e % MT) * 16, nn = (e / MT) * 8;
  const int r0 = (2 * z + 1) * N, c0 = 2 * z * N, row = lane >> 2, col = nn + (lane & 3) * 2;
  float* tm = tmp + z * N * DX_TMP;
  float acc[4];
  if (z < pairs) {
    dx_tile_product<N>(&X[(r0 + m) * DX_LD + c0], DX_LD, &X[c0 * DX_LD + c0 + nn], DX_LD, acc);
    *(float2*)&tm[(m + row) * DX_TMP + col] = make_float2(acc[0], acc[1]);
    *(float2*)&tm[(m + row + 8) * DX_TMP + col] = make_float2(acc[2], acc[3]);
  }
  __syncthreads();
  if (z < pairs) {
    dx_tile_product<N>(&X[(r0 + m) * DX_LD + r0], DX_LD, tm + nn, DX_TMP, acc);
    *(float2*)&X[(r0 + m + row) * DX_LD + c0 + col] = make_float2(-acc[0], -acc[1]);
    *(float2*)&X[(r0 + m + row + 8) * DX_LD + c0 + col] = make_float2(-acc[2], -acc[3]);
  }
  __syncthreads();
}

// 1 / sqrt(|row|^2 + eps) of the rows of a staged tile (still in the loading threads' registers), rows from `len` on: 0
template <int NP>
__device__ __forceinline__ void dx_row_norms(const DcTile<NP>& tile, float eps, int len, float* out) {
  constexpr int LANES = NP / 8;                               // neighbouring lanes that hold a row
#pragma unroll
  for (int it = 0; it < DcTile<NP>::IT; ++it) {
    const int i = it * DC_THREADS + threadIdx.x, t = i / LANES;
    if (i >= DcTile<NP>::UNITS) break;                        // (whole warps)
    const uint32_t u[4] = {tile.u[it].x, tile.u[it].y, tile.u[it].z, tile.u[it].w};
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float x0 = bf16_bits_to_f32(u[e] & 0xffffu), x1 = __uint_as_float(u[e] & 0xffff0000u);
      ss += x0 * x0 + x1 * x1;
    }
#pragma unroll
    for (int d = LANES / 2; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
    if (i % LANES == 0) out[t] = t < len ? 1.f / sqrtf(ss + eps) : 0.f;
  }
}

// 16 rows of X diag(f) against the columns of a staged tile [64][..] from its row 0 on: acc += (three bf16 terms) x tile
template <int NF>
__device__ __forceinline__ void dx_apply(const float* __restrict__ X, const float* __restrict__ f, int mt, const __nv_bfloat16* tile, int ld,
                                         float (&acc)[NF][4]) {
  const int lane = threadIdx.x & 31, r0 = mt * 16 + (lane >> 2);
#pragma unroll
  for (int i = 0; i < NF; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 1
  for (int st = 0; st <= mt; ++st) {
    uint32_t a[3][4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int rr = r0 + (e & 1) * 8, cc = st * 16 + (lane & 3) * 2 + (e >> 1) * 8;
      const float2 x = *(const float2*)&X[rr * DX_LD + cc], w = *(const float2*)&f[cc];
      uint32_t t[3];
      dc_terms<3>(x.x * w.x, x.y * w.y, t);
      a[0][e] = t[0], a[1][e] = t[1], a[2][e] = t[2];
    }
#pragma unroll
    for (int d = 0; d < NF / 2; ++d) {
      uint32_t bf[4];
      dc_ldmatrix_trans(bf, &tile[(st * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + d * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int z = 2; z >= 0; --z) {                          // the smallest term first
        dc_mma(acc[2 * d], a[z], bf[0], bf[1]);
        dc_mma(acc[2 * d + 1], a[z], bf[2], bf[3]);
      }
    }
  }
}

// grid (chunks, H, B).  NP: n rounded up to 16, 32, 64 or 128; PT: value columns worked on at a time.
template <int NP, int PT>
__global__ void __launch_bounds__(DC_THREADS, 2) delta_prepare_kernel(const DeltaChunkArgs A) {
  constexpr int LK = NP + 8, LV = PT + 8, PLANE = DC_L * LK;
  extern __shared__ __align__(16) unsigned char dx_smem[];
  float* X = (float*)dx_smem;                                 // [64][DX_LD]: L, then its inverse
  float* tmp = X + DC_L * DX_LD;                              // [32][DX_TMP]
  __nv_bfloat16* Ws = (__nv_bfloat16*)(tmp + 32 * DX_TMP);    // [2 terms][64][LK], then K right behind: the image that goes out
  __nv_bfloat16* Qs = Ws;                                     // the queries, until W is there
  __nv_bfloat16* Ks = Ws + 2 * PLANE;                         // [64][LK]
  __nv_bfloat16* Vs = Ks + PLANE;                             // [64][LV]
  __shared__ double G[DC_L];                                  // running sums of log decays,
  __shared__ float2 gf[DC_L];                                 // the same as the sum of two floats: differences keep their digits
  __shared__ __align__(8) float beta[DC_L], rk[DC_L], rq[DC_L], fw[DC_L];
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, g = h / (A.H / A.qk_heads), n = A.n, p = A.p;
  const int t0 = c * DC_L, len = min(DC_L, A.T - t0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const size_t m0 = (size_t)b * A.T + t0, j = ((size_t)b * A.H + h) * A.chunks + c;
  DcTile<PT> vt;
  {
    DcTile<NP> kt, qt;
    kt.load(A.k + m0 * A.k_stride + (size_t)g * n, A.k_stride, len, n);
    qt.load(A.q + m0 * A.q_stride + (size_t)g * n, A.q_stride, len, n);
    vt.load(A.v + m0 * A.v_stride + (size_t)h * p, A.v_stride, len, p);
    if (warp == 0) {
      double ld[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        ld[e] = t < len ? fmax((double)delta_log_decay(__bfloat162float(A.raw_a[(m0 + t) * A.gate_stride + h]), A.dt_bias[h], A.a_log[h]),
                               DC_LOG_MIN)
                        : 0.0;
      }
      dc_running_sums(ld, G);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const double v = G[2 * lane + e];
        const float hi = (float)v;
        gf[2 * lane + e] = make_float2(hi, (float)(v - hi));
      }
    } else if (warp <= 2) {
      const int t = tid - 32;
      beta[t] = t < len ? delta_strength(__bfloat162float(A.raw_b[(m0 + t) * A.gate_stride + h])) : 0.f;
    }
    kt.template store<false>(Ks, LK);
    qt.template store<false>(Qs, LK);
    vt.template store<false>(Vs, LV);
    dx_row_norms<NP>(kt, A.unit_eps, len, rk);
    dx_row_norms<NP>(qt, A.unit_eps, len, rq);
  }
  for (int i = tid; i < DC_L * 8; i += DC_THREADS) Ks[(i >> 3) * LK + NP + (i & 7)] = __float2bfloat16_rn(0.f);      // the image's pad
  __syncthreads();
  if (tid < DC_L) {
    const float eg = expf((float)G[tid]);
    fw[tid] = beta[tid] * rk[tid] * eg;
    A.sc.row[j * DC_L + tid] = eg * (A.qs * rq[tid]);
    A.sc.fac[j * DC_L + tid] = expf((float)(G[DC_L - 1] - G[tid])) * rk[tid];
    if (tid == 0) A.sc.tot[j * 4] = expf((float)G[DC_L - 1]);
  }
  // (the two warps of a scheduler get row tiles whose triangles add up to the same work)
  const int half = warp >> 2, mt = half ? 7 - warp : warp, r0 = mt * 16 + (lane >> 2);
  {   // L and A: 16 tokens of a warp against 32 keys, none that lie after all of them
    float sl[4][4], sa[4][4];
#pragma unroll
    for (int f = 0; f < 4; ++f) sl[f][0] = sl[f][1] = sl[f][2] = sl[f][3] = sa[f][0] = sa[f][1] = sa[f][2] = sa[f][3] = 0.f;
    if (half * 32 <= mt * 16) {
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {
        uint32_t kf[4], qf[4];
        const int at = (mt * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8;
        dc_ldmatrix(kf, &Ks[at]);
        dc_ldmatrix(qf, &Qs[at]);
#pragma unroll
        for (int d = 0; d < 2; ++d) {
          const int s0 = half * 32 + d * 16;
          if (s0 > mt * 16) break;
          uint32_t bf[4];
          dc_ldmatrix(bf, &Ks[(s0 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8]);
          dc_mma(sl[2 * d], kf, bf[0], bf[1]);
          dc_mma(sl[2 * d + 1], kf, bf[2], bf[3]);
          dc_mma(sa[2 * d], qf, bf[0], bf[1]);
          dc_mma(sa[2 * d + 1], qf, bf[2], bf[3]);
        }
      }
      const float bt[2] = {beta[r0] * rk[r0], beta[r0 + 8] * rk[r0 + 8]}, qt[2] = {A.qs * rq[r0], A.qs * rq[r0 + 8]};
      const float2 gt[2] = {gf[r0], gf[r0 + 8]};
      __nv_bfloat16* out = A.sc.A + j * 2 * DC_L * DC_L;
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int s = half * 32 + f * 8 + (lane & 3) * 2;
        if (half * 32 + f * 8 > mt * 16 + 15) break;
        const float2 gs[2] = {gf[s], gf[s + 1]};
        const float rs[2] = {rk[s], rk[s + 1]};
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = r0 + e * 8;
          float l[2], a[2];
#pragma unroll
          for (int z = 0; z < 2; ++z) {                       // zeros above the diagonal (L: on it too) of the diagonal blocks
            const float w = s + z <= t ? rs[z] * expf((gt[e].x - gs[z].x) + (gt[e].y - gs[z].y)) : 0.f;
            l[z] = s + z < t ? sl[f][2 * e + z] * (bt[e] * w) : 0.f;
            a[z] = sa[f][2 * e + z] * (qt[e] * w);
          }
          *(float2*)&X[t * DX_LD + s] = make_float2(l[0], l[1]);
          uint32_t at[2];
          dc_terms<2>(a[0], a[1], at);
          *(uint32_t*)&out[t * DC_L + s] = at[0];
          *(uint32_t*)&out[(DC_L + t) * DC_L + s] = at[1];
        }
      }
    }
  }
  __syncthreads();
  {   // the eight 8 x 8 blocks on the diagonal: a thread per column, read before any is written
    const int r = (tid >> 3) * 8, cc = tid & 7;
    float x[8];
    if (tid < DC_L)
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float v = i == cc ? 1.f : 0.f;
#pragma unroll
        for (int k = 0; k < i; ++k) v = fmaf(-X[(r + i) * DX_LD + r + k], x[k], v);
        x[i] = v;
      }
    __syncwarp();                                             // (a block's columns lie in one warp)
    if (tid < DC_L)
#pragma unroll
      for (int i = 0; i < 8; ++i) X[(r + i) * DX_LD + r + cc] = x[i];
    if (tid >= DC_L)                                          // the zeros beside the 16 x 16 blocks that the last merge reads
      for (int i = tid - DC_L; i < 512; i += DC_THREADS - DC_L) X[((i >> 8) * 32 + ((i >> 4) & 15)) * DX_LD + (i >> 8) * 32 + 16 + (i & 15)] = 0.f;
  }
  __syncthreads();
  dx_merge<8>(X, tmp, 4);
  dx_merge_mma<16>(X, tmp, 2);
  dx_merge_mma<32>(X, tmp, 1);
  if (half == 0) {                                            // four warps: W = X diag(b e^G r) K, 16 tokens each
    float acc[NP / 8][4];
    dx_apply<NP / 8>(X, fw, mt, Ks, LK, acc);
#pragma unroll
    for (int f = 0; f < NP / 8; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t w[2];
        dc_terms<2>(acc[f][2 * e], acc[f][2 * e + 1], w);
        const int at = (r0 + e * 8) * LK + f * 8 + (lane & 3) * 2;
        *(uint32_t*)&Ws[at] = w[0];
        *(uint32_t*)&Ws[PLANE + at] = w[1];
      }
  }
  float* U0 = A.sc.U0 + j * DC_L * p;
#pragma unroll 1
  for (int p0 = 0; p0 < p; p0 += PT) {                        // the other four: U_0 = X diag(b) V
    if (half == 1) {
      float acc[PT / 8][4];
      dx_apply<PT / 8>(X, beta, mt, Vs, LV, acc);
#pragma unroll
      for (int f = 0; f < PT / 8; ++f)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int col = p0 + f * 8 + (lane & 3) * 2;
          if (col < p) *(float2*)&U0[(size_t)(r0 + e * 8) * p + col] = make_float2(acc[f][2 * e], acc[f][2 * e + 1]);
        }
    }
    if (p0 + PT < p) {
      vt.load(A.v + m0 * A.v_stride + (size_t)h * p + p0 + PT, A.v_stride, len, p - p0 - PT);
      __syncthreads();
      vt.template store<false>(Vs, LV);
      __syncthreads();
    }
  }
  __syncthreads();
  uint4* out = (uint4*)(A.sc.WK + j * 3 * PLANE);
  for (int i = tid; i < 3 * PLANE / 8; i += DC_THREADS) out[i] = ((const uint4*)Ws)[i];      // (the pad columns of W are never read)
}

__device__ __forceinline__ void dx_cp_async16(void* smem, const void* gmem, bool valid) {
  const int bytes = valid ? 16 : 0;                           // 0: the 16 bytes are zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem)), "l"(gmem), "r"(bytes) : "memory");
}

// NF neighbouring 8-column fragments of a row-major [16][..] tile at `at` (leading dimension ld)
template <int NF>
__device__ __forceinline__ void dx_columns(uint32_t (&bf)[NF][2], const __nv_bfloat16* at, int ld) {
  const int lane = threadIdx.x & 31;
  const __nv_bfloat16* row = at + ((lane & 7) + ((lane >> 3) & 1) * 8) * ld;
  if constexpr (NF == 1) {
    dc_ldmatrix_trans2(bf[0][0], bf[0][1], row);
  } else {
#pragma unroll
    for (int d = 0; d < NF / 2; ++d) {
      uint32_t r[4];
      dc_ldmatrix_trans(r, row + d * 16 + (lane >> 4) * 8);
      bf[2 * d][0] = r[0], bf[2 * d][1] = r[1], bf[2 * d + 1][0] = r[2], bf[2 * d + 1][1] = r[3];
    }
  }
}

constexpr uint32_t DX_WAIT_LIMIT = 1u << 22;
__device__ int g_delta_chunk_error = 0;

__device__ __forceinline__ bool dx_wait(uint64_t* bar, uint32_t parity) {
  for (uint32_t i = 0; i < DX_WAIT_LIMIT; ++i)
    if (mbar_try_wait(bar, parity)) return true;
  atomicCAS(&g_delta_chunk_error, 0, 1);
  return false;
}

// row pitch of the pass kernel's column tiles: eight rows of a fragment in different banks
__host__ __device__ constexpr int dx_pitch(int pt) { return pt == 8 ? 24 : pt + 8; }

// grid (p tiles of PT, H, B).  The block's [n][PT] slice of the state lives in the accumulators of the state product (MW row groups
// of RT x 16 and NW column groups over the warps); per chunk it goes out in two bf16 terms, as the state before the chunk and, in shared
// memory, as the operand of W S.  W and K travel two chunks ahead of the products (one bulk
// copy each).
template <int NP, int PT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32, 1) delta_pass_kernel(const DeltaChunkArgs A) {
  constexpr int THREADS = WARPS * 32, LK = NP + 8, LU = dx_pitch(PT), PLANE = DC_L * LK, STAGE = 3 * PLANE;      // a stage: two terms of W, then K
  constexpr int RT = NP >= 64 ? 2 : 1, MW = NP / 16 / RT;     // row tiles a warp has of the state, warps along the rows
  constexpr int NW = (WARPS / MW) < (PT / 8) ? (WARPS / MW) : (PT / 8), NS = PT / 8 / NW, NU = PT / 8 / (WARPS / 4);
  extern __shared__ __align__(16) unsigned char dx_smem[];
  __nv_bfloat16* stages = (__nv_bfloat16*)dx_smem;            // [3 stages][3][64][LK]
  __nv_bfloat16* Ss = stages + 3 * STAGE;                     // [2 terms][NP][LU]
  __nv_bfloat16* Us = Ss + 2 * NP * LU;                       // [3 terms][64][LU]
  __shared__ __align__(8) uint64_t full[3];
  __shared__ int gave_up;
  const int p0 = blockIdx.x * PT, h = blockIdx.y, b = blockIdx.z, n = A.n, p = A.p, chunks = A.chunks;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const size_t bh = (size_t)b * A.H + h, j0 = bh * chunks;
  const bool fresh = A.pos_ids[0] == 0;
  // one thread asks for a chunk's image in one bulk copy; every wait for it is bounded
  auto load_stage = [&](int c, int st) {
    if (tid == 0 && c < chunks) {
      mbar_expect_tx(&full[st], STAGE * 2);
      bulk_load_1d(stages + st * STAGE, A.sc.WK + (j0 + c) * STAGE, STAGE * 2, &full[st]);
    }
  };
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&full[i], 1);
    fence_barrier_init();
    gave_up = 0;
  }
  __syncthreads();
  load_stage(0, 0);
  load_stage(1, 1);
  // product of W and the state: 16 tokens x NU fragments of columns a warp
  const int ut = (warp & 3) * 16 + (lane >> 2), uc = (warp >> 2) * (NU * 8);
  float2 un[NU][2];
  float fn[2], tn;
  auto load_next = [&](int c) {
    const float* U0 = A.sc.U0 + (j0 + c) * DC_L * p;
#pragma unroll
    for (int f = 0; f < NU; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = p0 + uc + f * 8 + (lane & 3) * 2;
        un[f][e] = col < p ? *(const float2*)&U0[(size_t)(ut + e * 8) * p + col] : make_float2(0.f, 0.f);
      }
    fn[0] = A.sc.fac[(j0 + c) * DC_L + ut], fn[1] = A.sc.fac[(j0 + c) * DC_L + ut + 8];
    tn = A.sc.tot[(j0 + c) * 4];
  };
  load_next(0);
  // state product: rows from sm on, columns from sc0 on
  const bool owner = warp < MW * NW;
  const int sm = (warp % MW) * RT * 16, sc0 = (warp / MW) * (PT / NW);
  float S[RT][NS][4];
  float* state = A.state + bh * n * p;
#pragma unroll
  for (int q = 0; q < RT * NS * 2; ++q) {
    const int i = q / (2 * NS), f = (q / 2) % NS, e = q % 2;
    const int row = sm + i * 16 + (lane >> 2) + e * 8, col = p0 + sc0 + f * 8 + (lane & 3) * 2;
    const bool in = owner && !fresh && row < n && col < p;
    const float2 s = in ? *(const float2*)&state[(size_t)row * p + col] : make_float2(0.f, 0.f);
    S[i][f][2 * e] = s.x, S[i][f][2 * e + 1] = s.y;
  }
  int st = 0;
  uint32_t phase = 0;
  for (int c = 0; c < chunks; ++c) {
    if (owner) {
#pragma unroll
      for (int q = 0; q < RT * NS * 2; ++q) {
        const int i = q / (2 * NS), f = (q / 2) % NS, e = q % 2;
        const int row = sm + i * 16 + (lane >> 2) + e * 8, cl = sc0 + f * 8 + (lane & 3) * 2;
        uint32_t t[2];
        dc_terms<2>(S[i][f][2 * e], S[i][f][2 * e + 1], t);
        *(uint32_t*)&Ss[row * LU + cl] = t[0];
        *(uint32_t*)&Ss[(NP + row) * LU + cl] = t[1];
      }
    }
    if (!dx_wait(&full[st], phase)) gave_up = 1;
    __syncthreads();
    if (gave_up) {                     // the copies in flight get time to land before the block leaves; the host sees the code
      for (int i = 0; i < 2048; ++i) __nanosleep(512);
      return;
    }
    load_stage(c + 2, st == 0 ? 2 : st - 1);                  // (the stage of the chunk before this one: its readers have met since)
    const __nv_bfloat16* Ws = stages + st * STAGE;
    const __nv_bfloat16* Ks = Ws + 2 * PLANE;
    float acc[3][NU][4];
#pragma unroll
    for (int z = 0; z < 3; ++z)
#pragma unroll
      for (int f = 0; f < NU; ++f) acc[z][f][0] = acc[z][f][1] = acc[z][f][2] = acc[z][f][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk) {
      uint32_t wh[4], wl[4], sh[NU][2], sl[NU][2];
      const int at = ((warp & 3) * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8;
      dc_ldmatrix(wh, &Ws[at]);
      dc_ldmatrix(wl, &Ws[PLANE + at]);
      dx_columns<NU>(sh, &Ss[kk * 16 * LU + uc], LU);
      dx_columns<NU>(sl, &Ss[(NP + kk * 16) * LU + uc], LU);
#pragma unroll
      for (int f = 0; f < NU; ++f) {
        dc_mma(acc[0][f], wh, sh[f][0], sh[f][1]);
        dc_mma(acc[1][f], wh, sl[f][0], sl[f][1]);
        dc_mma(acc[2][f], wl, sh[f][0], sh[f][1]);
      }
    }
    {   // the state before the chunk, as it now lies in shared memory
      __nv_bfloat16* out = A.sc.S + (j0 + c) * 2 * n * p + p0;
#pragma unroll
      for (int it = 0; it < (2 * NP * PT / 8 + THREADS - 1) / THREADS; ++it) {
        const int i = it * THREADS + tid, r = i / (PT / 8), cl = (i % (PT / 8)) * 8, z = r / NP, row = r % NP;
        if (i < 2 * NP * PT / 8 && row < n && p0 + cl < p) *(uint4*)&out[(size_t)(z * n + row) * p + cl] = *(const uint4*)&Ss[r * LU + cl];
      }
    }
    __nv_bfloat16* U = A.sc.U + (j0 + c) * 2 * DC_L * p + p0;
#pragma unroll
    for (int f = 0; f < NU; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = ut + e * 8, cl = uc + f * 8 + (lane & 3) * 2;
        const float u0 = un[f][e].x - (acc[0][f][2 * e] + (acc[1][f][2 * e] + acc[2][f][2 * e]));
        const float u1 = un[f][e].y - (acc[0][f][2 * e + 1] + (acc[1][f][2 * e + 1] + acc[2][f][2 * e + 1]));
        uint32_t tm[3], tu[2];
        dc_terms<3>(u0 * fn[e], u1 * fn[e], tm);
#pragma unroll
        for (int z = 0; z < 3; ++z) *(uint32_t*)&Us[(z * DC_L + t) * LU + cl] = tm[z];
        if (p0 + cl < p) {
          dc_terms<2>(u0, u1, tu);
          *(uint32_t*)&U[(size_t)t * p + cl] = tu[0];
          *(uint32_t*)&U[(size_t)(DC_L + t) * p + cl] = tu[1];
        }
      }
    const float w = tn;
    if (c + 1 < chunks) load_next(c + 1);
    __syncthreads();
    if (owner) {
      float add[2][RT][NS][4];                                // the smaller terms' products, chains of their own
#pragma unroll
      for (int q = 0; q < RT * NS * 4; ++q) {
        const int i = q / (4 * NS), f = (q / 4) % NS, e = q % 4;
        S[i][f][e] *= w, add[0][i][f][e] = add[1][i][f][e] = 0.f;
      }
#pragma unroll
      for (int kt = 0; kt < DC_L / 16; ++kt) {
        uint32_t af[RT][4];
#pragma unroll
        for (int i = 0; i < RT; ++i)
          dc_ldmatrix_trans(af[i], &Ks[(kt * 16 + (lane & 7) + (lane >> 4) * 8) * LK + sm + i * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
        for (int z = 0; z < 3; ++z) {
          uint32_t bf[NS][2];
          dx_columns<NS>(bf, &Us[(z * DC_L + kt * 16) * LU + sc0], LU);
#pragma unroll
          for (int i = 0; i < RT; ++i)
#pragma unroll
            for (int f = 0; f < NS; ++f)
              dc_mma(z == 0 ? S[i][f] : add[z - 1][i][f], af[i], bf[f][0], bf[f][1]);
        }
      }
#pragma unroll
      for (int q = 0; q < RT * NS * 4; ++q) {
        const int i = q / (4 * NS), f = (q / 4) % NS, e = q % 4;
        S[i][f][e] += add[0][i][f][e] + add[1][i][f][e];
      }
    }
    if (++st == 3) st = 0, phase ^= 1u;
  }
  if (owner)
#pragma unroll
    for (int q = 0; q < RT * NS * 2; ++q) {
      const int i = q / (2 * NS), f = (q / 2) % NS, e = q % 2;
      const int row = sm + i * 16 + (lane >> 2) + e * 8, col = p0 + sc0 + f * 8 + (lane & 3) * 2;
      if (row < n && col < p) *(float2*)&state[(size_t)row * p + col] = make_float2(S[i][f][2 * e], S[i][f][2 * e + 1]);
    }
}

// grid (chunks * p tiles of 64, H, B): y = diag(row) Q S + A U.  A warp owns 16 consecutive tokens and half of the block's columns.
constexpr int DX_PT = 64;
template <int NP>
__global__ void __launch_bounds__(DC_THREADS, 2) delta_read_kernel(const DeltaChunkArgs A, int ptiles) {
  constexpr int LK = NP + 8, LA = DC_L + 8, LV = DX_PT + 8, NF = DX_PT / 16, CU = DX_PT / 8;
  extern __shared__ __align__(16) unsigned char dx_smem[];
  __nv_bfloat16* Qs = (__nv_bfloat16*)dx_smem;                // [64][LK]
  __nv_bfloat16* As = Qs + DC_L * LK;                         // [2 terms][64][LA]
  __nv_bfloat16* Us = As + 2 * DC_L * LA;                     // [2 terms][64][LV]
  __nv_bfloat16* Ss = Us + 2 * DC_L * LV;                     // [2 terms][NP][LV]
  const int c = blockIdx.x / ptiles, p0 = (blockIdx.x - c * ptiles) * DX_PT, h = blockIdx.y, b = blockIdx.z, g = h / (A.H / A.qk_heads);
  const int n = A.n, p = A.p, t0 = c * DC_L, len = min(DC_L, A.T - t0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mt = warp < 4 ? warp : 7 - warp, c0 = (warp >> 2) * (DX_PT / 2);
  const size_t m0 = (size_t)b * A.T + t0, j = ((size_t)b * A.H + h) * A.chunks + c;
  const bool has_state = c > 0 || A.pos_ids[0] != 0;
  // first what the product with the state needs, then the rest
  if (has_state) {
    const __nv_bfloat16* Q = A.q + m0 * A.q_stride + (size_t)g * n;
    for (int i = tid; i < DC_L * (NP / 8); i += DC_THREADS) {
      const int r = i / (NP / 8), ch = (i % (NP / 8)) * 8;
      const bool in = r < len && ch < n;
      dx_cp_async16(Qs + r * LK + ch, Q + (in ? (size_t)r * A.q_stride + ch : 0), in);
    }
    const __nv_bfloat16* S = A.sc.S + j * 2 * n * p;
#pragma unroll
    for (int it = 0; it < 2 * NP * CU / DC_THREADS; ++it) {
      const int i = it * DC_THREADS + tid, z = i / (NP * CU), r = (i / CU) % NP, cl = (i % CU) * 8;
      const bool in = r < n && p0 + cl < p;
      dx_cp_async16(Ss + (z * NP + r) * LV + cl, S + (in ? (size_t)(z * n + r) * p + p0 + cl : 0), in);
    }
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const __nv_bfloat16* Ag = A.sc.A + j * 2 * DC_L * DC_L;
  const __nv_bfloat16* U = A.sc.U + j * 2 * DC_L * p;
#pragma unroll
  for (int it = 0; it < 2 * DC_L * 8 / DC_THREADS; ++it) {    // (blocks of A above the diagonal hold anything: they meet nothing)
    const int i = it * DC_THREADS + tid, r = i / 8, cl = (i % 8) * 8;
    dx_cp_async16(As + r * LA + cl, Ag + r * DC_L + cl, true);
  }
#pragma unroll
  for (int it = 0; it < 2 * DC_L * CU / DC_THREADS; ++it) {
    const int i = it * DC_THREADS + tid, r = i / CU, cl = (i % CU) * 8;
    const bool in = p0 + cl < p;
    dx_cp_async16(Us + r * LV + cl, U + (in ? (size_t)r * p + p0 + cl : 0), in);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const int r0 = mt * 16 + (lane >> 2);
  const float e0 = A.sc.row[j * DC_L + r0], e1 = A.sc.row[j * DC_L + r0 + 8];
  float o[NF][4];
#pragma unroll
  for (int f = 0; f < NF; ++f) o[f][0] = o[f][1] = o[f][2] = o[f][3] = 0.f;
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  if (has_state) {
    float lo[NF][4];                                          // the smaller term's product, a chain of its own
#pragma unroll
    for (int f = 0; f < NF; ++f) lo[f][0] = lo[f][1] = lo[f][2] = lo[f][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk) {
      uint32_t qf[4], sh[NF][2], sl[NF][2];
      dc_ldmatrix(qf, &Qs[(mt * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8]);
      dx_columns<NF>(sh, &Ss[kk * 16 * LV + c0], LV);
      dx_columns<NF>(sl, &Ss[(NP + kk * 16) * LV + c0], LV);
#pragma unroll
      for (int f = 0; f < NF; ++f) {
        dc_mma(o[f], qf, sh[f][0], sh[f][1]);
        dc_mma(lo[f], qf, sl[f][0], sl[f][1]);
      }
    }
#pragma unroll
    for (int f = 0; f < NF; ++f)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[f][e] = (o[f][e] + lo[f][e]) * (e < 2 ? e0 : e1);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if (mt * 16 >= len) return;
#pragma unroll
  for (int st = 0; st < DC_L / 16; ++st) {                    // 16 tokens' writes at a time, none that lie after all of the warp's
    if (st > mt) break;
    uint32_t ah[4], al[4], uh[NF][2], ul[NF][2];
    const int at = (mt * 16 + (lane & 15)) * LA + st * 16 + (lane >> 4) * 8;
    dc_ldmatrix(ah, &As[at]);
    dc_ldmatrix(al, &As[DC_L * LA + at]);
    dx_columns<NF>(uh, &Us[st * 16 * LV + c0], LV);
    dx_columns<NF>(ul, &Us[(DC_L + st * 16) * LV + c0], LV);
#pragma unroll
    for (int f = 0; f < NF; ++f) {
      dc_mma(o[f], al, uh[f][0], uh[f][1]);
      dc_mma(o[f], ah, ul[f][0], ul[f][1]);
      dc_mma(o[f], ah, uh[f][0], uh[f][1]);
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = r0 + e * 8;
    if (r >= len) continue;
    float* yr = A.y + (m0 + r) * (size_t)A.H * p + (size_t)h * p + p0 + c0;
#pragma unroll
    for (int f = 0; f < NF; ++f) {
      const int col = f * 8 + (lane & 3) * 2;
      if (p0 + c0 + col < p) *(float2*)(yr + col) = make_float2(o[f][2 * e], o[f][2 * e + 1]);
    }
  }
}

template <int NP, int PT, int WARPS>
static int delta_pass_launch(const DeltaChunkArgs& A, int B, cudaStream_t st) {
  constexpr int smem = (3 * 3 * DC_L * (NP + 8) + (2 * NP + 3 * DC_L) * dx_pitch(PT)) * 2;
  static bool sized = false;
  if (!sized) {
    LL_CUDA(cudaFuncSetAttribute(delta_pass_kernel<NP, PT, WARPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    sized = true;
  }
  delta_pass_kernel<NP, PT, WARPS><<<dim3((A.p + PT - 1) / PT, A.H, B), WARPS * 32, smem, st>>>(A);
  LL_LAUNCH_OK("delta_pass_kernel");
  return LL_OK;
}

template <int NP, int PT>
static int delta_prepare_launch(const DeltaChunkArgs& A, int B, cudaStream_t st) {
  constexpr int smem = (DC_L * DX_LD + 32 * DX_TMP) * 4 + DC_L * (3 * (NP + 8) + PT + 8) * 2;
  static bool sized = false;
  if (!sized) {
    LL_CUDA(cudaFuncSetAttribute(delta_prepare_kernel<NP, PT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    sized = true;
  }
  delta_prepare_kernel<NP, PT><<<dim3(A.chunks, A.H, B), DC_THREADS, smem, st>>>(A);
  LL_LAUNCH_OK("delta_prepare_kernel");
  return LL_OK;
}

template <int NP>
static int delta_chunked_launch(const DeltaChunkArgs& A, int B, cudaStream_t st) {
  constexpr int smem_r = (DC_L * (NP + 8) + 2 * DC_L * (DC_L + 8) + 2 * (DC_L + NP) * (DX_PT + 8)) * 2;
  static bool sized = false;
  if (!sized) {
    LL_CUDA(cudaFuncSetAttribute(delta_read_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_r));
    sized = true;
  }
  int rc = A.p <= 64 ? delta_prepare_launch<NP, 64>(A, B, st) : delta_prepare_launch<NP, 128>(A, B, st);
  if (rc != LL_OK) return rc;
  // the narrowest column tiles whose blocks run side by side: a block walks the chunks one after the other
  const long long heads = (long long)B * A.H;
  if (heads * ((A.p + 7) / 8) <= sm_count()) rc = delta_pass_launch<NP, 8, 4>(A, B, st);
  else if (heads * ((A.p + 15) / 16) <= sm_count()) rc = delta_pass_launch<NP, 16, 8>(A, B, st);
  else rc = delta_pass_launch<NP, 32, 8>(A, B, st);
  if (rc != LL_OK) return rc;
  const int ptiles = (A.p + DX_PT - 1) / DX_PT;
  delta_read_kernel<NP><<<dim3(A.chunks * ptiles, A.H, B), DC_THREADS, smem_r, st>>>(A, ptiles);
  LL_LAUNCH_OK("delta_read_kernel");
  return LL_OK;
}

}  // namespace llb

using namespace llb;

extern "C" {

int ll_delta_chunked_supported(int dtype, int T, int n, int p, int q_stride, int k_stride, int v_stride) {
  return dtype == LL_BF16 && T >= DC_L && n % 8 == 0 && n <= 128 && p % 8 == 0 && ((q_stride | k_stride | v_stride) & 7) == 0;
}

size_t ll_delta_chunked_scratch_bytes(int B, int T, int H, int n, int p) {
  const size_t np = n <= 16 ? 16 : n <= 32 ? 32 : n <= 64 ? 64 : 128;
  // fac, row, tot; U_0 and the terms of U; A; the terms of the state; the stage's image
  const size_t per = (size_t)(2 * DC_L + 4) * 4 + (size_t)DC_L * p * 8 + DC_L * DC_L * 4 + (size_t)n * p * 4 + 3 * (size_t)DC_L * (np + 8) * 2;
  return (size_t)B * H * ((T + DC_L - 1) / DC_L) * per;
}

// 0, or 1 when a bounded wait of the pass kernel ran out since the library was loaded.
int ll_delta_chunk_error(void) {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_delta_chunk_error, sizeof(int)) != cudaSuccess) return -1;
  return v;
}

int ll_delta_chunked(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const void* raw_a,
                     const void* raw_b, int gate_stride, int dtype, const float* dt_bias, const float* a_log, float unit_eps, float qs,
                     float* state, const int32_t* pos_ids, float* y, int B, int T, int H, int qk_heads, int n, int p, float* scratch,
                     ll_stream stream) {
  LL_CHECK_ARG(q && k && v && raw_a && raw_b && dt_bias && a_log && state && pos_ids && y && scratch, "delta_chunked: null pointer");
  LL_CHECK_ARG(B >= 0 && T >= 0 && H > 0 && qk_heads > 0 && H % qk_heads == 0 && n > 0 && p > 0 && gate_stride >= H,
               "bad delta_chunked arguments");
  if (B == 0 || T == 0) return LL_OK;
  const uintptr_t at = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)y | (uintptr_t)scratch;
  if (!ll_delta_chunked_supported(dtype, T, n, p, q_stride, k_stride, v_stride) || (at & 15) != 0 || B > 65535 || H > 65535) {
    set_error("delta_chunked: bf16, at least %d tokens, n and p in multiples of 8 (n up to 128), rows on 16-byte boundaries", DC_L);
    return LL_ERR_UNSUPPORTED;
  }
  DeltaChunkArgs A;
  A.q = (const __nv_bfloat16*)q, A.k = (const __nv_bfloat16*)k, A.v = (const __nv_bfloat16*)v;
  A.raw_a = (const __nv_bfloat16*)raw_a, A.raw_b = (const __nv_bfloat16*)raw_b;
  A.q_stride = q_stride, A.k_stride = k_stride, A.v_stride = v_stride, A.gate_stride = gate_stride;
  A.dt_bias = dt_bias, A.a_log = a_log, A.unit_eps = unit_eps, A.qs = qs, A.state = state, A.pos_ids = pos_ids, A.y = y;
  A.T = T, A.H = H, A.qk_heads = qk_heads, A.n = n, A.p = p, A.chunks = (T + DC_L - 1) / DC_L;
  const size_t cells = (size_t)B * H * A.chunks;
  A.sc.fac = scratch;
  A.sc.row = A.sc.fac + cells * DC_L;
  A.sc.tot = A.sc.row + cells * DC_L;
  A.sc.U0 = A.sc.tot + cells * 4;
  A.sc.A = (__nv_bfloat16*)(A.sc.U0 + cells * DC_L * p);
  A.sc.U = A.sc.A + cells * 2 * DC_L * DC_L;
  A.sc.S = A.sc.U + cells * 2 * DC_L * p;
  A.sc.WK = A.sc.S + cells * 2 * n * p;
  cudaStream_t st = (cudaStream_t)stream;
  if (n <= 16) return delta_chunked_launch<16>(A, B, st);
  if (n <= 32) return delta_chunked_launch<32>(A, B, st);
  if (n <= 64) return delta_chunked_launch<64>(A, B, st);
  return delta_chunked_launch<128>(A, B, st);
}

}  // extern "C"
