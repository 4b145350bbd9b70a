// What the recurrences that run in chunks of 64 tokens on tensor cores (decay_chunk.cu, delta_chunk.cu) share: fragments, fp32
// numbers as sums of bf16 terms, staging of activation rows, running sums of log decays.
#pragma once
#include "common.cuh"

namespace llb {

constexpr int DC_L = 64, DC_THREADS = 256;                   // tokens of a chunk
constexpr double DC_LOG_MIN = -1e4;                          // log of a decay of zero: e^-10000 is zero in fp32

__device__ __forceinline__ void dc_ldmatrix(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void dc_ldmatrix_trans(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void dc_ldmatrix_trans2(uint32_t& r0, uint32_t& r1, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(smem_u32(p)));
}
// D(16x8,f32) += A(16x16,bf16,row) * B(16x8,bf16,col); a function of registers alone, which the compiler may move between loads
__device__ __forceinline__ void dc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x as bf16 terms: the first of (a, b) packed, the rest left in a and b
__device__ __forceinline__ uint32_t dc_term(float& a, float& b) {
  const uint32_t u = pack_bf16(a, b);
  a -= bf16_bits_to_f32(u & 0xffffu), b -= __uint_as_float(u & 0xffff0000u);
  return u;
}
// The same of one pair, as all of its N terms, the largest first
template <int N>
__device__ __forceinline__ void dc_terms(float a, float b, uint32_t (&t)[N]) {
#pragma unroll
  for (int z = 0; z < N - 1; ++z) t[z] = dc_term(a, b);
  t[N - 1] = pack_bf16(a, b);
}
template <bool SILU>
__device__ __forceinline__ uint32_t dc_in2(uint32_t u) {
  if (!SILU) return u;
  return pack_bf16(silu_fast(bf16_bits_to_f32(u & 0xffffu)), silu_fast(__uint_as_float(u & 0xffff0000u)));
}
template <bool SILU>
__device__ __forceinline__ uint4 dc_in8(uint4 u) {
  return make_uint4(dc_in2<SILU>(u.x), dc_in2<SILU>(u.y), dc_in2<SILU>(u.z), dc_in2<SILU>(u.w));
}

// Rows of a [64][cols] slice of an activation matrix (cols a multiple of 8, at most PAD), requested: unit it of a thread is 16 bytes.
template <int PAD>
struct DcTile {
  static constexpr int UNITS = DC_L * (PAD / 8), IT = (UNITS + DC_THREADS - 1) / DC_THREADS;
  uint4 u[IT];
  __device__ __forceinline__ void load(const __nv_bfloat16* __restrict__ base, int stride, int len, int cols) {
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = it * DC_THREADS + threadIdx.x, s = i / (PAD / 8), ch = (i % (PAD / 8)) * 8;
      u[it] = make_uint4(0u, 0u, 0u, 0u);
      if (i < UNITS && s < len && ch < cols) u[it] = *(const uint4*)(base + (size_t)s * stride + ch);
    }
  }
  template <bool SILU>
  __device__ __forceinline__ void store(__nv_bfloat16* smem, int ld) const {
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = it * DC_THREADS + threadIdx.x, s = i / (PAD / 8), ch = (i % (PAD / 8)) * 8;
      if (i < UNITS) *(uint4*)&smem[s * ld + ch] = dc_in8<SILU>(u[it]);
    }
  }
};

// Running sums over a chunk's 64 numbers in fp64 by one warp, two neighbouring numbers a lane: G[t] = v_0 + ... + v_t
__device__ __forceinline__ void dc_running_sums(const double (&v)[2], double* G) {
  const int lane = threadIdx.x & 31;
  double incl = v[0] + v[1];
#pragma unroll
  for (int d = 1; d < 32; d <<= 1) {
    const double o = __shfl_up_sync(0xffffffffu, incl, d);
    if (lane >= d) incl += o;
  }
  G[2 * lane] = incl - v[1];
  G[2 * lane + 1] = incl;
}

}  // namespace llb
