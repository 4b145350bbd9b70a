// The gated delta rule of delta_rule.cu for prompts in bf16, on tensor cores.  Within a chunk of 64 tokens, S_0 the state before it,
// G_t the sum of the log decays up to token t, k^_t = r_t k_t the unit keys and b_t the write strengths, what token t writes is
//
//   u_t = b_t (v_t - e^(G_t) S_0^T k^_t - sum_(s < t) e^(G_t - G_s) (k^_s.k^_t) u_s),       S_t = e^(G_t) S_0 + sum_(s <= t) e^(G_t - G_s) k^_s u_s^T
//
// a triangular system (I + L) U = diag(b) (V - diag(e^G) K^ S_0) whose matrix does not depend on the state:
//
//   prepare   X = (I + L)^-1;   W = X diag(b e^G) K^,   U_0 = X diag(b) V                    (a block per chunk)
//   pass      U = U_0 - W S_c;   S_(c+1) = e^(G_last) S_c + sum_s e^(G_last - G_s) k^_s u_s^T       (a block per column tile of a head,
//             which walks the chunks with its slice of the state in registers)
//   read      y_t = q^_t.( e^(G_t) S_c ) + sum_(s <= t) e^(G_t - G_s) (q^_t.k^_s) u_s             (a block per chunk)
//
// X is formed by substitution (16 x 16 blocks, then by halves), which holds for any keys: a series in powers of L would not.  k, q and
// v are bf16 as they stand, the fp32 factors are split into bf16 terms (fp32 accumulation): three (24 bits) where X meets K and V
// and where U enters the state; two (16 bits, the three largest of the four products) where W meets the state and where the
// read-out's weights and the queries meet U and the state.  Sums of log decays are fp64.  The state handed on is fp32.
#include "chunk_mma.cuh"
#include "delta.cuh"

namespace llb {

constexpr int DX_LD = DC_L + 4;                              // row pitch of the fp32 triangles
constexpr int DX_TMP = 36;

struct DeltaScratch {       // per (sequence, head, chunk) j: G at j * 64, W at j * 2 * 64 * n, ...
  double* G;
  float* r;                 // 1 / |k|
  float* U;                 // [64][p]
  float* S;                 // [n][p], the state before the chunk
  __nv_bfloat16* W;         // [2 terms][64][n]
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

// A lower triangle's merge by halves: the blocks [r0 .. r0 + N)[c0 .. c0 + N) of the inverse, -X_22 (L_21 X_11), c0 = r0 - N.
// `pairs` merges side by side, a thread per four columns of a row (N * N / 4 threads a merge); two barriers.
template <int N>
__device__ __forceinline__ void dx_merge(const float* __restrict__ L, float* X, float* tmp, int pairs) {
  constexpr int TPM = N * N / 4;
  const int z = threadIdx.x / TPM, e = threadIdx.x - z * TPM, i = e / (N / 4), j = (e % (N / 4)) * 4;
  const int r0 = (2 * z + 1) * N, c0 = 2 * z * N;
  float* tm = tmp + z * N * DX_TMP;
  if (z < pairs) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int k = 0; k < N; ++k) fma4(o, L[(r0 + i) * DX_LD + c0 + k], *(const float4*)&X[(c0 + k) * DX_LD + c0 + j]);
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

// The fragment of rows r, r + 8 and columns c, c + 1, c + 8, c + 9 of X diag(f), as three bf16 terms
__device__ __forceinline__ void dx_fragment(const float* __restrict__ X, const float* __restrict__ f, int r, int c, uint32_t (&a)[3][4]) {
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int rr = r + (e & 1) * 8, cc = c + (e >> 1) * 8;
    const float2 x = *(const float2*)&X[rr * DX_LD + cc];
    uint32_t t[3];
    dc_terms<3>(x.x * f[cc], x.y * f[cc + 1], t);
    a[0][e] = t[0], a[1][e] = t[1], a[2][e] = t[2];
  }
}

// grid (chunks, H, B).  NP: n rounded up to 16, 32, 64 or 128.
template <int NP>
__global__ void __launch_bounds__(DC_THREADS, 3) delta_prepare_kernel(const DeltaChunkArgs A) {
  constexpr int LK = NP + 8, LV = 64 + 8, NF = NP >= 32 ? NP / 16 : 2;     // NF: 8-column fragments of a warp's share of the keys
  extern __shared__ __align__(16) unsigned char dx_smem[];
  float* X = (float*)dx_smem;                                 // [64][DX_LD]
  float* L = X + DC_L * DX_LD;                                // [64][DX_LD], below the diagonal
  float* tmp = L + DC_L * DX_LD;                              // [32][DX_TMP]
  __nv_bfloat16* Ks = (__nv_bfloat16*)(tmp + 32 * DX_TMP);    // [64][LK]
  __nv_bfloat16* Vs = Ks + DC_L * LK;                         // [64][LV]
  __shared__ double G[DC_L];
  __shared__ float beta[DC_L], rk[DC_L], fw[DC_L];
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, g = h / (A.H / A.qk_heads), n = A.n, p = A.p;
  const int t0 = c * DC_L, len = min(DC_L, A.T - t0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const size_t m0 = (size_t)b * A.T + t0, j = ((size_t)b * A.H + h) * A.chunks + c;
  DcTile<NP> kt;
  DcTile<64> vt;
  kt.load(A.k + m0 * A.k_stride + (size_t)g * n, A.k_stride, len, n);
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
  } else if (warp <= 2) {
    const int t = tid - 32;
    beta[t] = t < len ? delta_strength(__bfloat162float(A.raw_b[(m0 + t) * A.gate_stride + h])) : 0.f;
  }
  kt.template store<false>(Ks, LK);
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 8; ++e) {                               // a warp's eight rows: 1 / |k|
    const int t = warp * 8 + e;
    float ss = 0.f;
    for (int i = 2 * lane; i < NP; i += 64) {
      const uint32_t u = *(const uint32_t*)&Ks[t * LK + i];
      const float x0 = bf16_bits_to_f32(u & 0xffffu), x1 = bf16_bits_to_f32(u >> 16);
      ss += x0 * x0 + x1 * x1;
    }
    ss = warp_sum(ss);
    if (lane == 0) rk[t] = t < len ? 1.f / sqrtf(ss + A.unit_eps) : 0.f;
  }
  __syncthreads();
  if (tid < DC_L) {
    fw[tid] = beta[tid] * rk[tid] * expf((float)G[tid]);
    A.sc.G[j * DC_L + tid] = G[tid];
    A.sc.r[j * DC_L + tid] = rk[tid];
  }
  const int mt = warp & 3, half = warp >> 2, r0 = mt * 16 + (lane >> 2);
  {   // L: 16 tokens of a warp against 32 keys, none that lie after all of them
    float sc[4][4];
#pragma unroll
    for (int f = 0; f < 4; ++f) sc[f][0] = sc[f][1] = sc[f][2] = sc[f][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk) {
      uint32_t af[4];
      dc_ldmatrix(af, &Ks[(mt * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int d = 0; d < 2; ++d) {
        const int s0 = half * 32 + d * 16;
        if (s0 > mt * 16) break;
        uint32_t bf[4];
        dc_ldmatrix(bf, &Ks[(s0 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8]);
        mma_bf16_16816(sc[2 * d], af[0], af[1], af[2], af[3], bf[0], bf[1]);
        mma_bf16_16816(sc[2 * d + 1], af[0], af[1], af[2], af[3], bf[2], bf[3]);
      }
    }
#pragma unroll
    for (int f = 0; f < 4; ++f)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = r0 + (e >> 1) * 8, s = half * 32 + f * 8 + (lane & 3) * 2 + (e & 1);
        if (s < t) L[t * DX_LD + s] = sc[f][e] * (beta[t] * rk[t] * rk[s] * expf((float)(G[t] - G[s])));
      }
  }
  __syncthreads();
  if (tid < DC_L) {   // the four 16 x 16 blocks on the diagonal: a thread per column
    const int r = (tid >> 4) * 16, cc = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float v = i == cc ? 1.f : 0.f;
#pragma unroll
      for (int k = 0; k < i; ++k) v = fmaf(-L[(r + i) * DX_LD + r + k], x[k], v);
      x[i] = v;
      X[(r + i) * DX_LD + r + cc] = v;
    }
  } else {            // meanwhile the zeros right of them that the merge of the halves reads
    for (int i = tid - DC_L; i < 512; i += DC_THREADS - DC_L) {
      const int r = (i >> 8) * 32 + ((i >> 4) & 15), cc = (i >> 8) * 32 + 16 + (i & 15);
      X[r * DX_LD + cc] = 0.f;
    }
  }
  __syncthreads();
  dx_merge<16>(L, X, tmp, 2);
  dx_merge<32>(L, X, tmp, 1);
  // W = X diag(b e^G r) K: a warp's 16 tokens x half of the key columns, as two bf16 terms
  if (NP >= 32 || half == 0) {
    const int c0 = NP >= 32 ? half * (NP / 2) : 0;
    float acc[NF][4];
#pragma unroll
    for (int f = 0; f < NF; ++f) acc[f][0] = acc[f][1] = acc[f][2] = acc[f][3] = 0.f;
#pragma unroll 1
    for (int st = 0; st <= mt; ++st) {
      uint32_t af[3][4];
      dx_fragment(X, fw, r0, st * 16 + (lane & 3) * 2, af);
#pragma unroll
      for (int d = 0; d < NF / 2; ++d) {
        uint32_t bf[4];
        dc_ldmatrix_trans(bf, &Ks[(st * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LK + c0 + d * 16 + (lane >> 4) * 8]);
#pragma unroll
        for (int z = 2; z >= 0; --z) {
          mma_bf16_16816(acc[2 * d], af[z][0], af[z][1], af[z][2], af[z][3], bf[0], bf[1]);
          mma_bf16_16816(acc[2 * d + 1], af[z][0], af[z][1], af[z][2], af[z][3], bf[2], bf[3]);
        }
      }
    }
    __nv_bfloat16* W = A.sc.W + j * 2 * DC_L * n;
#pragma unroll
    for (int f = 0; f < NF; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = r0 + e * 8, col = c0 + f * 8 + (lane & 3) * 2;
        if (col >= n) continue;
        uint32_t w[2];
        dc_terms<2>(acc[f][2 * e], acc[f][2 * e + 1], w);
        *(uint32_t*)&W[(size_t)t * n + col] = w[0];
        *(uint32_t*)&W[(size_t)(DC_L + t) * n + col] = w[1];
      }
  }
  // U_0 = X diag(b) V, 64 value columns at a time
  float* U = A.sc.U + j * DC_L * p;
#pragma unroll 1
  for (int p0 = 0; p0 < p; p0 += 64) {
    vt.template store<false>(Vs, LV);
    __syncthreads();
    if (p0 + 64 < p) vt.load(A.v + m0 * A.v_stride + (size_t)h * p + p0 + 64, A.v_stride, len, p - p0 - 64);
    float acc[4][4];
#pragma unroll
    for (int f = 0; f < 4; ++f) acc[f][0] = acc[f][1] = acc[f][2] = acc[f][3] = 0.f;
#pragma unroll 1
    for (int st = 0; st <= mt; ++st) {
      uint32_t af[3][4];
      dx_fragment(X, beta, r0, st * 16 + (lane & 3) * 2, af);
#pragma unroll
      for (int d = 0; d < 2; ++d) {
        uint32_t bf[4];
        dc_ldmatrix_trans(bf, &Vs[(st * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LV + half * 32 + d * 16 + (lane >> 4) * 8]);
#pragma unroll
        for (int z = 2; z >= 0; --z) {
          mma_bf16_16816(acc[2 * d], af[z][0], af[z][1], af[z][2], af[z][3], bf[0], bf[1]);
          mma_bf16_16816(acc[2 * d + 1], af[z][0], af[z][1], af[z][2], af[z][3], bf[2], bf[3]);
        }
      }
    }
#pragma unroll
    for (int f = 0; f < 4; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = p0 + half * 32 + f * 8 + (lane & 3) * 2;
        if (col < p) *(float2*)&U[(size_t)(r0 + e * 8) * p + col] = make_float2(acc[f][2 * e], acc[f][2 * e + 1]);
      }
    __syncthreads();
  }
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

// grid (p tiles of PT, H, B).  The block's [n][PT] slice of the state lives in the accumulators of the state product (MW row tiles of
// 16 x NW column groups over the warps); per chunk it goes out as the state before the chunk and, in two bf16 terms, to shared
// memory as the operand of W S.  W and K of the next chunk are copied under the current chunk's products.
template <int NP, int PT>
__global__ void __launch_bounds__(DC_THREADS, 1) delta_pass_kernel(const DeltaChunkArgs A) {
  constexpr int LK = NP + 8, LU = PT + 8, STAGE = 3 * DC_L * LK;           // a stage: two terms of W, then K
  constexpr int MW = NP / 16, NW = (8 / MW) < (PT / 8) ? (8 / MW) : (PT / 8), NS = PT / 8 / NW, NU = PT / 16;
  extern __shared__ __align__(16) unsigned char dx_smem[];
  __nv_bfloat16* stages = (__nv_bfloat16*)dx_smem;            // [2 stages][3][64][LK]
  __nv_bfloat16* Ss = stages + 2 * STAGE;                     // [2 terms][NP][LU]
  __nv_bfloat16* Us = Ss + 2 * NP * LU;                       // [3 terms][64][LU]
  __shared__ float fac[2][DC_L], tot[2];
  const int p0 = blockIdx.x * PT, h = blockIdx.y, b = blockIdx.z, g = h / (A.H / A.qk_heads), n = A.n, p = A.p, chunks = A.chunks;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const size_t bh = (size_t)b * A.H + h;
  const bool fresh = A.pos_ids[0] == 0;
  // columns n .. NP of every staged row are never copied: zeros
  for (int i = tid; i < 2 * 3 * DC_L * (NP - n); i += DC_THREADS) {
    const int r = i / (NP - n);
    stages[r * LK + n + i - r * (NP - n)] = __float2bfloat16_rn(0.f);
  }
  auto load_stage = [&](int c, int st) {
    const int len = min(DC_L, A.T - c * DC_L), per = n / 8;
    const __nv_bfloat16* W = A.sc.W + (bh * chunks + c) * 2 * DC_L * n;
    const __nv_bfloat16* K = A.k + ((size_t)b * A.T + c * DC_L) * A.k_stride + (size_t)g * n;
    __nv_bfloat16* dst = stages + st * STAGE;
    for (int i = tid; i < 3 * DC_L * per; i += DC_THREADS) {
      const int r = i / per, ch = (i - r * per) * 8, s = r - 2 * DC_L;
      if (s < 0) dx_cp_async16(dst + r * LK + ch, W + (size_t)r * n + ch, true);
      else dx_cp_async16(dst + r * LK + ch, K + (size_t)(s < len ? s : 0) * A.k_stride + ch, s < len);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_stage(0, 0);
  // product of W and the state: 16 tokens x PT / 2 columns a warp
  const int ut = (warp & 3) * 16 + (lane >> 2), uc = (warp >> 2) * (PT / 2);
  float2 un[NU][2];
  auto load_u = [&](int c) {
    const float* U = A.sc.U + (bh * chunks + c) * DC_L * p;
#pragma unroll
    for (int f = 0; f < NU; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = p0 + uc + f * 8 + (lane & 3) * 2;
        un[f][e] = col < p ? *(const float2*)&U[(size_t)(ut + e * 8) * p + col] : make_float2(0.f, 0.f);
      }
  };
  double gl = 0.0, gt = 0.0;
  float rt = 0.f;
  auto load_fac = [&](int c) {
    if (tid < DC_L) {
      const size_t j = bh * chunks + c;
      gl = A.sc.G[j * DC_L + DC_L - 1], gt = A.sc.G[j * DC_L + tid], rt = A.sc.r[j * DC_L + tid];
    }
  };
  auto store_fac = [&](int st) {
    if (tid < DC_L) {
      fac[st][tid] = expf((float)(gl - gt)) * rt;
      if (tid == 0) tot[st] = expf((float)gl);
    }
  };
  load_u(0);
  load_fac(0);
  store_fac(0);
  // state product: row tile sm, column group sg
  const bool owner = warp < MW * NW;
  const int sm = warp % MW, sc0 = (warp / MW) * (PT / NW), srow = sm * 16 + (lane >> 2);
  float S[NS][4];
  float* state = A.state + bh * n * p;
#pragma unroll
  for (int f = 0; f < NS; ++f)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int row = srow + e * 8, col = p0 + sc0 + f * 8 + (lane & 3) * 2;
      const bool in = owner && !fresh && row < n && col < p;
      const float2 s = in ? *(const float2*)&state[(size_t)row * p + col] : make_float2(0.f, 0.f);
      S[f][2 * e] = s.x, S[f][2 * e + 1] = s.y;
    }
  for (int c = 0; c < chunks; ++c) {
    const int st = c & 1;
    if (owner) {
      float* out = A.sc.S + (bh * chunks + c) * n * p;
#pragma unroll
      for (int f = 0; f < NS; ++f)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int row = srow + e * 8, cl = sc0 + f * 8 + (lane & 3) * 2;
          if (row < n && p0 + cl < p) *(float2*)&out[(size_t)row * p + p0 + cl] = make_float2(S[f][2 * e], S[f][2 * e + 1]);
          uint32_t t[2];
          dc_terms<2>(S[f][2 * e], S[f][2 * e + 1], t);
          *(uint32_t*)&Ss[row * LU + cl] = t[0];
          *(uint32_t*)&Ss[(NP + row) * LU + cl] = t[1];
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (c + 1 < chunks) {
      load_stage(c + 1, st ^ 1);
      load_fac(c + 1);
    }
    const __nv_bfloat16* Ws = stages + st * STAGE;
    const __nv_bfloat16* Ks = Ws + 2 * DC_L * LK;
    {
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
        dc_ldmatrix(wl, &Ws[DC_L * LK + at]);
        dx_columns<NU>(sh, &Ss[kk * 16 * LU + uc], LU);
        dx_columns<NU>(sl, &Ss[(NP + kk * 16) * LU + uc], LU);
#pragma unroll
        for (int f = 0; f < NU; ++f) {
          mma_bf16_16816(acc[0][f], wh[0], wh[1], wh[2], wh[3], sh[f][0], sh[f][1]);
          mma_bf16_16816(acc[1][f], wh[0], wh[1], wh[2], wh[3], sl[f][0], sl[f][1]);
          mma_bf16_16816(acc[2][f], wl[0], wl[1], wl[2], wl[3], sh[f][0], sh[f][1]);
        }
      }
      float* U = A.sc.U + (bh * chunks + c) * DC_L * p;
#pragma unroll
      for (int f = 0; f < NU; ++f)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = ut + e * 8, cl = uc + f * 8 + (lane & 3) * 2;
          const float u0 = un[f][e].x - (acc[0][f][2 * e] + (acc[1][f][2 * e] + acc[2][f][2 * e]));
          const float u1 = un[f][e].y - (acc[0][f][2 * e + 1] + (acc[1][f][2 * e + 1] + acc[2][f][2 * e + 1]));
          if (p0 + cl < p) *(float2*)&U[(size_t)t * p + p0 + cl] = make_float2(u0, u1);
          uint32_t tm[3];
          dc_terms<3>(u0 * fac[st][t], u1 * fac[st][t], tm);
#pragma unroll
          for (int z = 0; z < 3; ++z) *(uint32_t*)&Us[(z * DC_L + t) * LU + cl] = tm[z];
        }
    }
    if (c + 1 < chunks) {
      load_u(c + 1);
      store_fac(st ^ 1);
    }
    __syncthreads();
    if (owner) {
      const float w = tot[st];
#pragma unroll
      for (int f = 0; f < NS; ++f) S[f][0] *= w, S[f][1] *= w, S[f][2] *= w, S[f][3] *= w;
#pragma unroll
      for (int kt = 0; kt < DC_L / 16; ++kt) {
        uint32_t af[4];
        dc_ldmatrix_trans(af, &Ks[(kt * 16 + (lane & 7) + (lane >> 4) * 8) * LK + sm * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
        for (int z = 2; z >= 0; --z) {
          uint32_t bf[NS][2];
          dx_columns<NS>(bf, &Us[(z * DC_L + kt * 16) * LU + sc0], LU);
#pragma unroll
          for (int f = 0; f < NS; ++f) mma_bf16_16816(S[f], af[0], af[1], af[2], af[3], bf[f][0], bf[f][1]);
        }
      }
    }
  }
  if (owner)
#pragma unroll
    for (int f = 0; f < NS; ++f)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = srow + e * 8, col = p0 + sc0 + f * 8 + (lane & 3) * 2;
        if (row < n && col < p) *(float2*)&state[(size_t)row * p + col] = make_float2(S[f][2 * e], S[f][2 * e + 1]);
      }
}

// grid (chunks * p tiles of 64, H, B).  A warp owns 16 consecutive tokens and half of the block's columns; its queries come from
// global memory straight into fragments.
constexpr int DX_PT = 64;
template <int NP>
__global__ void __launch_bounds__(DC_THREADS, 2) delta_read_kernel(const DeltaChunkArgs A, int ptiles) {
  constexpr int LK = NP + 8, LV = DX_PT + 8, NF = DX_PT / 16;
  extern __shared__ __align__(16) unsigned char dx_smem[];
  __nv_bfloat16* Ks = (__nv_bfloat16*)dx_smem;                // [64][LK]
  __nv_bfloat16* Us = Ks + DC_L * LK;                         // [2 terms][64][LV]
  __nv_bfloat16* Ss = Us + 2 * DC_L * LV;                     // [2 terms][NP][LV]
  __shared__ double G[DC_L];
  __shared__ float rk[DC_L];
  const int c = blockIdx.x / ptiles, p0 = (blockIdx.x - c * ptiles) * DX_PT, h = blockIdx.y, b = blockIdx.z, g = h / (A.H / A.qk_heads);
  const int n = A.n, p = A.p, t0 = c * DC_L, len = min(DC_L, A.T - t0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, row0 = (warp & 3) * 16, c0 = (warp >> 2) * (DX_PT / 2);
  const size_t m0 = (size_t)b * A.T + t0, j = ((size_t)b * A.H + h) * A.chunks + c;
  const bool has_state = c > 0 || A.pos_ids[0] != 0;
  const float* S = A.sc.S + j * n * p;
  const float* U = A.sc.U + j * DC_L * p;
  DcTile<NP> kt;
  kt.load(A.k + m0 * A.k_stride + (size_t)g * n, A.k_stride, len, n);
  constexpr int CU = DX_PT / 4, IU = DC_L * CU / DC_THREADS, IS = NP * CU / DC_THREADS;     // 16-byte units of a thread: U, state
  float4 uv[IU], sv[IS];
#pragma unroll
  for (int it = 0; it < IU; ++it) {
    const int i = it * DC_THREADS + tid, r = i / CU, col = p0 + (i % CU) * 4;
    uv[it] = col < p ? *(const float4*)&U[(size_t)r * p + col] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (has_state)
#pragma unroll
    for (int it = 0; it < IS; ++it) {
      const int i = it * DC_THREADS + tid, r = i / CU, col = p0 + (i % CU) * 4;
      sv[it] = (r < n && col < p) ? *(const float4*)&S[(size_t)r * p + col] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  if (tid < DC_L) G[tid] = A.sc.G[j * DC_L + tid], rk[tid] = A.sc.r[j * DC_L + tid];
  // query fragments: rows (lane / 4) and + 8 of the warp's 16, columns (lane % 4) * 2 and + 8 of every 16; |q|^2 of both rows
  uint32_t qf[NP / 16][4];
  const int r0 = row0 + (lane >> 2);
#pragma unroll
  for (int kk = 0; kk < NP / 16; ++kk)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = r0 + (e & 1) * 8, col = kk * 16 + (lane & 3) * 2 + (e >> 1) * 8;
      qf[kk][e] = (r < len && col < n) ? *(const uint32_t*)(A.q + (m0 + r) * A.q_stride + (size_t)g * n + col) : 0u;
    }
  auto store_terms = [&](__nv_bfloat16* dst, int plane, int i, float4 f) {
    const int r = i / CU, col = (i % CU) * 4;
    const uint32_t h0 = dc_term(f.x, f.y), h1 = dc_term(f.z, f.w);
    *(uint2*)&dst[r * LV + col] = make_uint2(h0, h1);
    *(uint2*)&dst[plane + r * LV + col] = make_uint2(pack_bf16(f.x, f.y), pack_bf16(f.z, f.w));
  };
  kt.template store<false>(Ks, LK);
#pragma unroll
  for (int it = 0; it < IU; ++it) store_terms(Us, DC_L * LV, it * DC_THREADS + tid, uv[it]);
  if (has_state)
#pragma unroll
    for (int it = 0; it < IS; ++it) store_terms(Ss, NP * LV, it * DC_THREADS + tid, sv[it]);
  float qq[2] = {0.f, 0.f};
#pragma unroll
  for (int kk = 0; kk < NP / 16; ++kk)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float x0 = bf16_bits_to_f32(qf[kk][e] & 0xffffu), x1 = bf16_bits_to_f32(qf[kk][e] >> 16);
      qq[e & 1] += x0 * x0 + x1 * x1;
    }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    qq[e] += __shfl_xor_sync(0xffffffffu, qq[e], 1);
    qq[e] += __shfl_xor_sync(0xffffffffu, qq[e], 2);
    qq[e] = A.qs / sqrtf(qq[e] + A.unit_eps);
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
      for (int z = 1; z >= 0; --z) {
        uint32_t bf[NF][2];
        dx_columns<NF>(bf, &Ss[(z * NP + kk * 16) * LV + c0], LV);
#pragma unroll
        for (int f = 0; f < NF; ++f) mma_bf16_16816(o[f], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], bf[f][0], bf[f][1]);
      }
    const float e0 = expf((float)g0), e1 = expf((float)g1);
#pragma unroll
    for (int f = 0; f < NF; ++f) o[f][0] *= e0, o[f][1] *= e0, o[f][2] *= e1, o[f][3] *= e1;
  }
#pragma unroll
  for (int st = 0; st < DC_L / 16; ++st) {                    // 16 tokens' writes at a time, none that lie after all of the warp's
    if (st * 16 > row0) break;
    float sc[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk) {
      uint32_t bf[4];
      dc_ldmatrix(bf, &Ks[(st * 16 + (lane & 7) + (lane >> 4) * 8) * LK + kk * 16 + ((lane >> 3) & 1) * 8]);
      mma_bf16_16816(sc[0], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], bf[0], bf[1]);
      mma_bf16_16816(sc[1], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], bf[2], bf[3]);
    }
    uint32_t ah[4], al[4];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int s = st * 16 + i * 8 + (lane & 3) * 2 + (e & 1), r = r0 + (e >> 1) * 8;
        sc[i][e] = s <= r ? sc[i][e] * (expf((float)((e >> 1 ? g1 : g0) - G[s])) * rk[s]) : 0.f;
      }
      ah[2 * i] = dc_term(sc[i][0], sc[i][1]), al[2 * i] = pack_bf16(sc[i][0], sc[i][1]);
      ah[2 * i + 1] = dc_term(sc[i][2], sc[i][3]), al[2 * i + 1] = pack_bf16(sc[i][2], sc[i][3]);
    }
    uint32_t uh[NF][2], ul[NF][2];
    dx_columns<NF>(uh, &Us[st * 16 * LV + c0], LV);
    dx_columns<NF>(ul, &Us[(DC_L + st * 16) * LV + c0], LV);
#pragma unroll
    for (int f = 0; f < NF; ++f) {
      mma_bf16_16816(o[f], al[0], al[1], al[2], al[3], uh[f][0], uh[f][1]);
      mma_bf16_16816(o[f], ah[0], ah[1], ah[2], ah[3], ul[f][0], ul[f][1]);
      mma_bf16_16816(o[f], ah[0], ah[1], ah[2], ah[3], uh[f][0], uh[f][1]);
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
      if (p0 + c0 + col < p) *(float2*)(yr + col) = make_float2(o[f][2 * e] * qq[e], o[f][2 * e + 1] * qq[e]);
    }
  }
}

template <int NP, int PT>
static int delta_pass_launch(const DeltaChunkArgs& A, int B, cudaStream_t st) {
  constexpr int smem = (2 * 3 * DC_L * (NP + 8) + (2 * NP + 3 * DC_L) * (PT + 8)) * 2;
  static bool sized = false;
  if (!sized) {
    LL_CUDA(cudaFuncSetAttribute(delta_pass_kernel<NP, PT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    sized = true;
  }
  delta_pass_kernel<NP, PT><<<dim3((A.p + PT - 1) / PT, A.H, B), DC_THREADS, smem, st>>>(A);
  LL_LAUNCH_OK("delta_pass_kernel");
  return LL_OK;
}

template <int NP>
static int delta_chunked_launch(const DeltaChunkArgs& A, int B, cudaStream_t st) {
  constexpr int smem_p = (2 * DC_L * DX_LD + 32 * DX_TMP) * 4 + DC_L * (NP + 8 + 64 + 8) * 2;
  constexpr int smem_r = (DC_L * (NP + 8) + 2 * (DC_L + NP) * (DX_PT + 8)) * 2;
  static bool sized = false;
  if (!sized) {
    LL_CUDA(cudaFuncSetAttribute(delta_prepare_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_p));
    LL_CUDA(cudaFuncSetAttribute(delta_read_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_r));
    sized = true;
  }
  delta_prepare_kernel<NP><<<dim3(A.chunks, A.H, B), DC_THREADS, smem_p, st>>>(A);
  LL_LAUNCH_OK("delta_prepare_kernel");
  // narrow column tiles until there is a block for most of the SMs
  const long long wide = (long long)B * A.H * ((A.p + 31) / 32);
  const int rc = wide * 3 >= 2 * sm_count() ? delta_pass_launch<NP, 32>(A, B, st) : delta_pass_launch<NP, 16>(A, B, st);
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
  const size_t per = (size_t)DC_L * (sizeof(double) + sizeof(float)) + ((size_t)DC_L * (n + p) + (size_t)n * p) * sizeof(float);
  return (size_t)B * H * ((T + DC_L - 1) / DC_L) * per;
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
  A.sc.G = (double*)scratch;
  A.sc.r = (float*)(A.sc.G + cells * DC_L);
  A.sc.U = A.sc.r + cells * DC_L;
  A.sc.S = A.sc.U + cells * DC_L * p;
  A.sc.W = (__nv_bfloat16*)(A.sc.S + cells * n * p);
  cudaStream_t st = (cudaStream_t)stream;
  if (n <= 16) return delta_chunked_launch<16>(A, B, st);
  if (n <= 32) return delta_chunked_launch<32>(A, B, st);
  if (n <= 64) return delta_chunked_launch<64>(A, B, st);
  return delta_chunked_launch<128>(A, B, st);
}

}  // extern "C"
