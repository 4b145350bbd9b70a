// A residual stream kept in fp32 whatever the activation dtype: scaled embedding rows, the
// "norm on the sublayer's output" update with a one-number RMSNorm gain, the weighted sum over
// the outputs of all earlier layers (depth-weighted average), and the gated-linear-unit
// activation with clamped pre-activations that the feed-forward layers of such models use.
//
// Every kernel takes the activation dtype as a template parameter (the GEMMs between these ops
// read and write that dtype) and does its arithmetic in fp32.
#include "common.cuh"

namespace llb {

// Block-wide sum of one float per thread (any blockDim.x that is a multiple of 32, up to 1024).
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if (lane == 0) red[w] = v;
  __syncthreads();
  float t = (threadIdx.x < nw) ? red[threadIdx.x] : 0.f;
  if (w == 0) {
    t = warp_sum(t);
    if (lane == 0) red[0] = t;
  }
  __syncthreads();
  t = red[0];
  __syncthreads();
  return t;
}

// x[m][:] = wte[idx[m]][:] * scale  (fp32), and the same rounded to the activation dtype.
template <typename TW, typename TA>
__global__ void embed_scaled_kernel(const TW* __restrict__ wte, const int64_t* __restrict__ idx, float scale,
                                    float* __restrict__ x, TA* __restrict__ x_act, int dim) {
  const int m = blockIdx.x;
  const TW* row = wte + (size_t)idx[m] * dim;
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    const float v = dt<TW>::ld(row, i) * scale;
    x[(size_t)m * dim + i] = v;
    if (x_act) dt<TA>::st(x_act, (size_t)m * dim + i, v);
  }
}

// r = x + gain * y / sqrt(mean(y^2) + eps)                      -> out      (fp32; may be a slot of `stack`)
// n_mix > 0:  v = mix_w[n_mix-1] * r + sum_{j < n_mix-1} mix_w[j] * stack[j]   else v = r
// v -> next (fp32, optional) and next_act (activation dtype, optional)
// x == nullptr means a plain norm (r = gain * y / rms).
template <typename TY, typename TA>
__global__ void gain_norm_add_mix_kernel(const float* x, const TY* __restrict__ y,
                                         const float* __restrict__ gain, float eps, float* out,
                                         const float* stack, size_t stack_stride,
                                         const float* __restrict__ mix_w, int n_mix, float* next,
                                         TA* __restrict__ next_act, int dim) {
  __shared__ float red[32];
  const size_t base = (size_t)blockIdx.x * dim;
  float ss = 0.f;
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    const float v = dt<TY>::ld(y, base + i);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float k = gain[0] / sqrtf(ss / (float)dim + eps);
  const float w_last = n_mix > 0 ? mix_w[n_mix - 1] : 1.f;
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    float r = dt<TY>::ld(y, base + i) * k;
    if (x) r += x[base + i];
    if (out) out[base + i] = r;
    float v = r * w_last;
    for (int j = 0; j < n_mix - 1; ++j) v += mix_w[j] * stack[(size_t)j * stack_stride + base + i];
    if (next) next[base + i] = v;
    if (next_act) dt<TA>::st(next_act, base + i, v);
  }
}

// Eight neighbouring numbers of an activation row as fp32 (16-byte accesses in bf16, two in fp32).
template <typename T> __device__ __forceinline__ void ld8(const T* p, float (&o)[8]);
template <> __device__ __forceinline__ void ld8<float>(const float* p, float (&o)[8]) {
  const float4 a = ((const float4*)p)[0], b = ((const float4*)p)[1];
  o[0] = a.x, o[1] = a.y, o[2] = a.z, o[3] = a.w, o[4] = b.x, o[5] = b.y, o[6] = b.z, o[7] = b.w;
}
template <> __device__ __forceinline__ void ld8<__nv_bfloat16>(const __nv_bfloat16* p, float (&o)[8]) {
  const uint4 u = *(const uint4*)p;
  o[0] = bf16_bits_to_f32(u.x & 0xffffu), o[1] = bf16_bits_to_f32(u.x >> 16);
  o[2] = bf16_bits_to_f32(u.y & 0xffffu), o[3] = bf16_bits_to_f32(u.y >> 16);
  o[4] = bf16_bits_to_f32(u.z & 0xffffu), o[5] = bf16_bits_to_f32(u.z >> 16);
  o[6] = bf16_bits_to_f32(u.w & 0xffffu), o[7] = bf16_bits_to_f32(u.w >> 16);
}
template <typename T> __device__ __forceinline__ void st8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void st8<float>(float* p, const float (&v)[8]) {
  ((float4*)p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  ((float4*)p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void st8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  uint32_t k[4];
#pragma unroll
  for (int q = 0; q < 4; ++q) k[q] = (uint32_t)f32_to_bf16_bits(v[2 * q]) | ((uint32_t)f32_to_bf16_bits(v[2 * q + 1]) << 16);
  *(uint4*)p = make_uint4(k[0], k[1], k[2], k[3]);
}

// Gated linear unit with clamped pre-activations, on the output of one GEMM over the stacked
// [gate; up] weight:  g = min(gu[m][c], limit), u = clamp(gu[m][ff + c], -limit, limit),
// h[m][c] = g * sigmoid(alpha * g) * (u + shift).
__device__ __forceinline__ float glu_unit(float g, float u, float limit, float alpha, float shift) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + shift);
}
// bias (optional): fp32 [2 ff], added to [gate | up] before the clamps; rows of h lie h_stride apart
template <typename T>
__global__ void glu_unit_kernel(const T* __restrict__ gu, int gu_stride, int ff, const float* __restrict__ bias, float limit, float alpha,
                                float shift, T* __restrict__ h, int h_stride, size_t n) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const size_t m = i / ff;
  const int c = (int)(i - m * ff);
  float g = dt<T>::ld(gu, m * gu_stride + c), u = dt<T>::ld(gu, m * gu_stride + ff + c);
  if (bias) g += bias[c], u += bias[ff + c];
  dt<T>::st(h, m * h_stride + c, glu_unit(g, u, limit, alpha, shift));
}
// ff, gu_stride multiples of 8 and 16-byte aligned rows: a thread owns eight columns of one row
template <typename T>
__global__ void glu_unit8_kernel(const T* __restrict__ gu, int gu_stride, int ff, const float* __restrict__ bias, float limit, float alpha,
                                 float shift, T* __restrict__ h, int h_stride, int n8) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n8) return;
  const int per = ff / 8, m = i / per, c = (i - m * per) * 8;
  const T* row = gu + (size_t)m * gu_stride + c;
  float g[8], u[8];
  ld8<T>(row, g);
  ld8<T>(row + ff, u);
  if (bias) {
    float bg[8], bu[8];
    ld8<float>(bias + c, bg);
    ld8<float>(bias + ff + c, bu);
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] += bg[e], u[e] += bu[e];
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) g[e] = glu_unit(g[e], u[e], limit, alpha, shift);
  st8<T>(h + (size_t)m * h_stride + c, g);
}

template <typename T>
static int glu_unit_launch(const void* gu, int gu_stride, int ff, const float* bias, float limit, float alpha, float shift, void* h,
                           int h_stride, int rows, cudaStream_t st) {
  const size_t n = (size_t)rows * ff;
  if (ff % 8 == 0 && gu_stride % 8 == 0 && h_stride % 8 == 0 && (((uintptr_t)gu | (uintptr_t)h | (uintptr_t)bias) & 15) == 0 &&
      n / 8 < (1ull << 31)) {
    const int n8 = (int)(n / 8);
    glu_unit8_kernel<T><<<(n8 + 127) / 128, 128, 0, st>>>((const T*)gu, gu_stride, ff, bias, limit, alpha, shift, (T*)h, h_stride, n8);
  } else {
    glu_unit_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, st>>>((const T*)gu, gu_stride, ff, bias, limit, alpha, shift, (T*)h, h_stride,
                                                                    n);
  }
  LL_LAUNCH_OK("glu_unit_kernel");
  return LL_OK;
}

}  // namespace llb

using namespace llb;

extern "C" {

int ll_embed_scaled(const void* wte, int wte_dtype, const int64_t* idx, float scale, float* x, void* x_act,
                    int act_dtype, int M, int dim, ll_stream stream) {
  LL_CHECK_ARG(wte && idx && x && M >= 0 && dim > 0, "bad embed_scaled arguments");
  if (M == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int threads = dim >= 1024 ? 256 : 128;
  if (wte_dtype == LL_F32 && act_dtype == LL_F32)
    embed_scaled_kernel<float, float><<<M, threads, 0, st>>>((const float*)wte, idx, scale, x, (float*)x_act, dim);
  else if (wte_dtype == LL_BF16 && act_dtype == LL_BF16)
    embed_scaled_kernel<__nv_bfloat16, __nv_bfloat16><<<M, threads, 0, st>>>((const __nv_bfloat16*)wte, idx, scale, x,
                                                                            (__nv_bfloat16*)x_act, dim);
  else if (wte_dtype == LL_BF16 && act_dtype == LL_F32)
    embed_scaled_kernel<__nv_bfloat16, float><<<M, threads, 0, st>>>((const __nv_bfloat16*)wte, idx, scale, x, (float*)x_act, dim);
  else {
    set_error("embed_scaled: unsupported dtypes %d / %d", wte_dtype, act_dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("embed_scaled_kernel");
  return LL_OK;
}

int ll_gain_norm_add_mix(const float* x, const void* y, int y_dtype, const float* gain, float eps, float* out,
                         const float* stack, size_t stack_stride, const float* mix_w, int n_mix, float* next,
                         void* next_act, int act_dtype, int rows, int dim, ll_stream stream) {
  LL_CHECK_ARG(y && gain && rows >= 0 && dim > 0 && n_mix >= 0, "bad gain_norm_add_mix arguments");
  LL_CHECK_ARG(n_mix <= 1 || (stack && mix_w), "gain_norm_add_mix: a mix needs the stack and its weights");
  LL_CHECK_ARG(n_mix == 0 || mix_w, "gain_norm_add_mix: a mix needs its weights");
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int threads = dim >= 2048 ? 512 : dim >= 512 ? 256 : 128;
  if (y_dtype == LL_F32 && act_dtype == LL_F32)
    gain_norm_add_mix_kernel<float, float><<<rows, threads, 0, st>>>(x, (const float*)y, gain, eps, out, stack, stack_stride,
                                                                     mix_w, n_mix, next, (float*)next_act, dim);
  else if (y_dtype == LL_BF16 && act_dtype == LL_BF16)
    gain_norm_add_mix_kernel<__nv_bfloat16, __nv_bfloat16><<<rows, threads, 0, st>>>(
        x, (const __nv_bfloat16*)y, gain, eps, out, stack, stack_stride, mix_w, n_mix, next, (__nv_bfloat16*)next_act, dim);
  else if (y_dtype == LL_F32 && act_dtype == LL_BF16)
    gain_norm_add_mix_kernel<float, __nv_bfloat16><<<rows, threads, 0, st>>>(x, (const float*)y, gain, eps, out, stack, stack_stride,
                                                                             mix_w, n_mix, next, (__nv_bfloat16*)next_act, dim);
  else {
    set_error("gain_norm_add_mix: unsupported dtypes %d / %d", y_dtype, act_dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("gain_norm_add_mix_kernel");
  return LL_OK;
}

int ll_glu_unit_rows(const void* gu, int gu_stride, int ff, const float* bias, float limit, float alpha, float shift, void* h,
                     int h_stride, int dtype, int rows, ll_stream stream) {
  LL_CHECK_ARG(gu && h && ff > 0 && gu_stride >= 2 * ff && h_stride >= ff && rows >= 0, "bad glu_unit arguments");
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == LL_F32) return glu_unit_launch<float>(gu, gu_stride, ff, bias, limit, alpha, shift, h, h_stride, rows, st);
  if (dtype == LL_BF16) return glu_unit_launch<__nv_bfloat16>(gu, gu_stride, ff, bias, limit, alpha, shift, h, h_stride, rows, st);
  set_error("glu_unit: unsupported dtype %d", dtype);
  return LL_ERR_UNSUPPORTED;
}

int ll_glu_unit(const void* gu, int gu_stride, int ff, float limit, float alpha, float shift, void* h, int dtype, int rows,
                ll_stream stream) {
  return ll_glu_unit_rows(gu, gu_stride, ff, nullptr, limit, alpha, shift, h, ff, dtype, rows, stream);
}

int ll_glu_clamp(const void* gu, int gu_stride, int ff, float limit, float alpha, void* h, int dtype, int rows,
                 ll_stream stream) {
  return ll_glu_unit(gu, gu_stride, ff, limit, alpha, 1.f, h, dtype, rows, stream);
}

}  // extern "C"

// ---- two-branch layers on an fp32 stream: x += sum of branch outputs, then two norms of the same x -----------------
namespace llb {

// x[m][:] += s0 * a0 + s1 * a1 + s2 * a2 (each optional, activation dtype TA), in place, fp32.  Then, with
// n = x / sqrt(mean(x^2) + eps):  out1 = n * w1 (fp32 or TA, see out1_f32; optional), out2 = n * w2 (TA; optional).
template <typename TA>
__global__ void add_norm_pair_kernel(float* __restrict__ x, const TA* __restrict__ a0, float s0, const TA* __restrict__ a1,
                                     float s1, const TA* __restrict__ a2, float s2, const float* __restrict__ w1,
                                     const float* __restrict__ w2, float eps, void* __restrict__ out1, int out1_f32,
                                     TA* __restrict__ out2, int dim) {
  __shared__ float red[32];
  const size_t base = (size_t)blockIdx.x * dim;
  float ss = 0.f;
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    float v = x[base + i];
    if (a0 || a1 || a2) {
      float add = 0.f;
      if (a0) add += s0 * dt<TA>::ld(a0, base + i);
      if (a1) add += s1 * dt<TA>::ld(a1, base + i);
      if (a2) add += s2 * dt<TA>::ld(a2, base + i);
      v += add;
      x[base + i] = v;
    }
    ss += v * v;
  }
  if (!out1 && !out2) return;
  ss = block_sum(ss, red);
  const float k = 1.f / sqrtf(ss / (float)dim + eps);
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    const float n = x[base + i] * k;
    if (out1) {
      if (out1_f32) ((float*)out1)[base + i] = n * w1[i];
      else dt<TA>::st((TA*)out1, base + i, n * w1[i]);
    }
    if (out2) dt<TA>::st(out2, base + i, n * w2[i]);
  }
}

// x[m][:] += s * (a + a_bias) + step, in place, fp32 (a: optional, activation dtype TA, with an optional fp32 bias row; step: an
// optional fp32 row).  Then, if asked for, the norm of the same row: the layer norm out = (x - mean) / sqrt(var + eps) * w + b, var
// the mean of the squared deviations (formed from the deviations themselves, in a second sweep over the row the block holds), or
// (RMS) out = x / sqrt(mean(x^2) + eps) * w.  One block per row; VPT > 0: the row stays in registers, VPT runs of four numbers per
// thread; VPT = 0: any length, the row in shared memory.
template <typename TA> __device__ __forceinline__ float4 ld4(const TA* p);
template <> __device__ __forceinline__ float4 ld4<float>(const float* p) { return *(const float4*)p; }
template <> __device__ __forceinline__ float4 ld4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 u = *(const uint2*)p;
  return make_float4(bf16_bits_to_f32(u.x & 0xffffu), bf16_bits_to_f32(u.x >> 16), bf16_bits_to_f32(u.y & 0xffffu),
                     bf16_bits_to_f32(u.y >> 16));
}
template <typename TA> __device__ __forceinline__ void st4(TA* p, float4 v);
template <> __device__ __forceinline__ void st4<float>(float* p, float4 v) { *(float4*)p = v; }
template <> __device__ __forceinline__ void st4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  *(uint2*)p = make_uint2((uint32_t)f32_to_bf16_bits(v.x) | ((uint32_t)f32_to_bf16_bits(v.y) << 16),
                          (uint32_t)f32_to_bf16_bits(v.z) | ((uint32_t)f32_to_bf16_bits(v.w) << 16));
}

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }

template <typename TA, int VPT, bool RMS>
__global__ void add_row_norm_kernel(float* __restrict__ x, const TA* __restrict__ a, float s, const float* __restrict__ a_bias,
                                    const float* __restrict__ step, const float* __restrict__ w, const float* __restrict__ b, float eps,
                                    TA* __restrict__ out, int dim) {
  extern __shared__ float ln_row[];
  __shared__ float red[32];
  const size_t base = (size_t)blockIdx.x * dim;
  float sum = 0.f;
  if constexpr (VPT > 0) {
    float4 v[VPT > 0 ? VPT : 1], av[VPT > 0 ? VPT : 1];
    const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 4;
      v[k] = i < dim ? *(const float4*)(x + base + i) : zero4;
      if (a) av[k] = i < dim ? ld4<TA>(a + base + i) : zero4;
    }
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 4;
      if (a) {
        if (a_bias && i < dim) av[k] = add4(av[k], *(const float4*)(a_bias + i));
        v[k].x += s * av[k].x, v[k].y += s * av[k].y, v[k].z += s * av[k].z, v[k].w += s * av[k].w;
      }
      if (step && i < dim) v[k] = add4(v[k], *(const float4*)(step + i));
      if ((a || step) && i < dim) *(float4*)(x + base + i) = v[k];
      if (!RMS) sum += (v[k].x + v[k].y) + (v[k].z + v[k].w);
    }
    if (!out) return;
    if constexpr (!RMS) {
      const float mean = block_sum(sum, red) / (float)dim;
#pragma unroll
      for (int k = 0; k < VPT; ++k) v[k].x -= mean, v[k].y -= mean, v[k].z -= mean, v[k].w -= mean;
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
      if ((k * blockDim.x + threadIdx.x) * 4 < dim) ss += (v[k].x * v[k].x + v[k].y * v[k].y) + (v[k].z * v[k].z + v[k].w * v[k].w);
    const float kn = 1.f / sqrtf(block_sum(ss, red) / (float)dim + eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 4;
      if (i < dim) {
        const float4 wv = *(const float4*)(w + i), bv = RMS ? zero4 : *(const float4*)(b + i);
        st4<TA>(out + base + i, make_float4(v[k].x * kn * wv.x + bv.x, v[k].y * kn * wv.y + bv.y, v[k].z * kn * wv.z + bv.z,
                                            v[k].w * kn * wv.w + bv.w));
      }
    }
  } else {
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
      float v = x[base + i];
      if (a) v += s * (dt<TA>::ld(a, base + i) + (a_bias ? a_bias[i] : 0.f));
      if (step) v += step[i];
      if (a || step) x[base + i] = v;
      ln_row[i] = v;
      sum += v;
    }
    if (!out) return;
    const float mean = RMS ? 0.f : block_sum(sum, red) / (float)dim;
    float ss = 0.f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {      // (a thread reads back what it wrote itself)
      const float d = ln_row[i] - mean;
      ss += d * d;
    }
    const float kn = 1.f / sqrtf(block_sum(ss, red) / (float)dim + eps);
    for (int i = threadIdx.x; i < dim; i += blockDim.x) dt<TA>::st(out, base + i, (ln_row[i] - mean) * kn * w[i] + (RMS ? 0.f : b[i]));
  }
}

template <typename TA, bool RMS>
static int add_row_norm_launch(float* x, const void* a, float s, const float* a_bias, const float* step, const float* w, const float* b,
                               float eps, void* out, int rows, int dim, cudaStream_t st) {
  const bool vec = dim % 4 == 0 && dim <= 8192 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)b | (uintptr_t)a | (uintptr_t)out |
                                                    (uintptr_t)a_bias | (uintptr_t)step) & 15) == 0;
#define LL_ALN(VPT, NT, SM) \
  add_row_norm_kernel<TA, VPT, RMS><<<rows, NT, SM, st>>>(x, (const TA*)a, s, a_bias, step, w, b, eps, (TA*)out, dim)
  if (vec) {
    if (dim <= 2048) LL_ALN(1, (dim / 4 + 31) / 32 * 32, 0);
    else if (dim <= 4096) LL_ALN(2, 512, 0);
    else LL_ALN(4, 512, 0);
  } else {
    const size_t smem = (size_t)dim * sizeof(float);
    if (smem > 200 * 1024) {
      set_error("add + norm: rows of %d numbers", dim);
      return LL_ERR_UNSUPPORTED;
    }
    static bool sized = false;
    if (!sized && smem > 48 * 1024) {
      LL_CUDA(cudaFuncSetAttribute(add_row_norm_kernel<TA, 0, RMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
      sized = true;
    }
    LL_ALN(0, dim >= 512 ? 256 : 128, smem);
  }
#undef LL_ALN
  LL_LAUNCH_OK("add_row_norm_kernel");
  return LL_OK;
}

// RMS norm of an fp32 row in `groups` equal parts (each by its own root mean square), a weight, and a gate (silu, or a
// sigmoid when gate_sigmoid):
//   gate_first: t = y * gate(g);  out = t / rms_part(t) * w          (the gate enters the norm)
//   otherwise : out = y / rms_part(y) * w * gate(g)                  (the gate follows the norm)
// w has C entries, or C / groups entries shared by the parts (w_shared).  One block per row.
// A part of y spans y_gs >= C / groups numbers (the rest is skipped), except with `stab`: then number C / groups of every
// part is a normaliser's product nq and stab[m][part] a stabiliser mx, and the part is first divided by
// max(|nq|, exp(-mx)) + 1e-6 (the read-out of a matrix memory with exponential gates).
template <typename TA>
__global__ void gated_group_norm_kernel(const float* __restrict__ y, int y_gs, const float* __restrict__ stab,
                                        const TA* __restrict__ gate, int gate_stride, const float* __restrict__ w, int w_shared,
                                        float eps, int groups, int gate_first, int gate_sigmoid, TA* __restrict__ out, int out_stride, int C) {
  const int m = blockIdx.x;
  const int gs = C / groups;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  for (int g = warp; g < groups; g += nw) {
    const float* yr = y + ((size_t)m * groups + g) * y_gs;
    const TA* gr = gate + (size_t)m * gate_stride + (size_t)g * gs;
    const float pre = stab ? 1.f / (fmaxf(fabsf(yr[gs]), expf(-stab[(size_t)m * groups + g])) + 1e-6f) : 1.f;
    float ss = 0.f;
    for (int i = lane; i < gs; i += 32) {
      float v = yr[i] * pre;
      if (gate_first) {
        const float z = dt<TA>::ld(gr, i);
        v *= (gate_sigmoid ? 1.f : z) / (1.f + expf(-z));
      }
      ss += v * v;
    }
    ss = warp_sum(ss);
    const float k = 1.f / sqrtf(ss / (float)gs + eps);
    for (int i = lane; i < gs; i += 32) {
      const float z = dt<TA>::ld(gr, i);
      const float sg = (gate_sigmoid ? 1.f : z) / (1.f + expf(-z));
      const float wv = w[w_shared ? i : g * gs + i];
      const float yv = yr[i] * pre;
      const float v = gate_first ? (yv * sg) * k * wv : yv * k * wv * sg;
      dt<TA>::st(out, (size_t)m * out_stride + (size_t)g * gs + i, v);
    }
  }
}

// The same for short parts in multiples of four numbers without a normaliser: a warp per (row, part), VPT float4 a lane, the part in
// registers between the two sweeps.
template <typename TA, int VPT>
__global__ void __launch_bounds__(256) gated_group_norm4_kernel(const float* __restrict__ y, int y_gs, const TA* __restrict__ gate,
                                                                int gate_stride, const float* __restrict__ w, int w_shared, float eps,
                                                                int groups, int gate_first, int gate_sigmoid, TA* __restrict__ out,
                                                                int out_stride, int gs, int parts) {
  const int part = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (part >= parts) return;
  const int m = part / groups, g = part - m * groups;
  const float* yr = y + (size_t)part * y_gs;
  const TA* gr = gate + (size_t)m * gate_stride + (size_t)g * gs;
  const float* wr = w + (w_shared ? 0 : (size_t)g * gs);
  float4 v[VPT], z[VPT];
  float ss = 0.f;
  auto gated = [&](float t) { return (gate_sigmoid ? 1.f : t) / (1.f + expf(-t)); };
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * 32 + lane) * 4;
    v[k] = i < gs ? *(const float4*)(yr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    z[k] = i < gs ? ld4<TA>(gr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    z[k] = make_float4(gated(z[k].x), gated(z[k].y), gated(z[k].z), gated(z[k].w));
    const float4 t = make_float4(v[k].x * z[k].x, v[k].y * z[k].y, v[k].z * z[k].z, v[k].w * z[k].w);
    const float4 n = gate_first ? t : v[k];
    ss += (n.x * n.x + n.y * n.y) + (n.z * n.z + n.w * n.w);
    v[k] = t;
  }
  const float kn = 1.f / sqrtf(warp_sum(ss) / (float)gs + eps);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * 32 + lane) * 4;
    if (i >= gs) continue;
    const float4 wv = *(const float4*)(wr + i);
    st4<TA>(out + (size_t)m * out_stride + (size_t)g * gs + i, make_float4(v[k].x * kn * wv.x, v[k].y * kn * wv.y, v[k].z * kn * wv.z,
                                                                          v[k].w * kn * wv.w));
  }
}

template <typename TA>
static int gated_group_norm4_launch(const float* y, int y_gs, const void* gate, int gate_stride, const float* w, int w_shared, float eps,
                                    int groups, int gate_first, int gate_sigmoid, void* out, int out_stride, int rows, int gs,
                                    cudaStream_t st) {
  const int parts = rows * groups;
#define LL_GGN4(VPT)                                                                                                                  \
  gated_group_norm4_kernel<TA, VPT><<<(parts + 7) / 8, 256, 0, st>>>(y, y_gs, (const TA*)gate, gate_stride, w, w_shared, eps, groups, \
                                                                     gate_first, gate_sigmoid, (TA*)out, out_stride, gs, parts)
  if (gs <= 128) LL_GGN4(1);
  else LL_GGN4(2);
#undef LL_GGN4
  LL_LAUNCH_OK("gated_group_norm4_kernel");
  return LL_OK;
}

// The same for long parts (a whole row of heads normed together): a block per (row, part), the gated numbers of the first sweep
// kept in shared memory.  V numbers at a time per thread (4: rows and parts on 4-number boundaries).
template <typename TA, int V>
__global__ void gated_group_norm_wide_kernel(const float* __restrict__ y, const TA* __restrict__ gate, int gate_stride,
                                             const float* __restrict__ w, int w_shared, float eps, int gate_first, int gate_sigmoid,
                                             TA* __restrict__ out, int out_stride, int gs) {
  extern __shared__ __align__(16) float ggn_row[];
  __shared__ float red[32];
  const size_t m = blockIdx.y;
  const int g = blockIdx.x, groups = gridDim.x;
  const float* yr = y + (m * groups + g) * gs;
  const TA* gr = gate + m * gate_stride + (size_t)g * gs;
  const float* wr = w + (w_shared ? 0 : (size_t)g * gs);
  TA* orow = out + m * out_stride + (size_t)g * gs;
  float ss = 0.f;
  auto gated = [&](float v, float z) {
    const float t = v * (gate_sigmoid ? 1.f : z) / (1.f + expf(-z));
    ss += gate_first ? t * t : v * v;
    return t;
  };
#pragma unroll 4
  for (int i = threadIdx.x * V; i < gs; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 v = *(const float4*)(yr + i), z = ld4<TA>(gr + i);
      *(float4*)(ggn_row + i) = make_float4(gated(v.x, z.x), gated(v.y, z.y), gated(v.z, z.z), gated(v.w, z.w));
    } else {
      ggn_row[i] = gated(yr[i], dt<TA>::ld(gr, i));
    }
  }
  const float k = 1.f / sqrtf(block_sum(ss, red) / (float)gs + eps);
#pragma unroll 4
  for (int i = threadIdx.x * V; i < gs; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 t = *(const float4*)(ggn_row + i), wv = *(const float4*)(wr + i);
      st4<TA>(orow + i, make_float4(t.x * k * wv.x, t.y * k * wv.y, t.z * k * wv.z, t.w * k * wv.w));
    } else {
      dt<TA>::st(orow, i, ggn_row[i] * k * wr[i]);
    }
  }
}

template <typename TA>
static int gated_group_norm_wide_launch(const float* y, const void* gate, int gate_stride, const float* w, int w_shared, float eps,
                                        int groups, int gate_first, int gate_sigmoid, void* out, int out_stride, int rows, int gs, cudaStream_t st) {
  const bool vec = ((gs | gate_stride | out_stride) & 3) == 0 && (((uintptr_t)y | (uintptr_t)w | (uintptr_t)out | (uintptr_t)gate) & (4 * sizeof(TA) - 1)) == 0 &&
                   (((uintptr_t)y | (uintptr_t)w) & 15) == 0;
  // few blocks: a thread's share of the row is what the launch takes
  int nt = (long long)rows * groups < 2 * sm_count() ? 1024 : 256;
  while (nt > 64 && nt * (vec ? 4 : 1) > gs) nt /= 2;
  const size_t smem = (size_t)gs * sizeof(float);
#define LL_GGN(V)                                                                                                                     \
  gated_group_norm_wide_kernel<TA, V><<<dim3(groups, rows), nt, smem, st>>>(y, (const TA*)gate, gate_stride, w, w_shared, eps, gate_first, \
                                                                            gate_sigmoid, (TA*)out, out_stride, gs)
  if (vec) LL_GGN(4);
  else LL_GGN(1);
#undef LL_GGN
  LL_LAUNCH_OK("gated_group_norm_wide_kernel");
  return LL_OK;
}

// in place: relu(v)^2
template <typename T>
__global__ void relu_squared_kernel(T* __restrict__ h, size_t n) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float v = fmaxf(dt<T>::ld(h, i), 0.f);
  dt<T>::st(h, i, v * v);
}

template <typename T>
__global__ void relu_squared8_kernel(T* __restrict__ h, size_t n8) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n8) return;
  float v[8];
  ld8<T>(h + i * 8, v);
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    const float r = fmaxf(v[e], 0.f);
    v[e] = r * r;
  }
  st8<T>(h + i * 8, v);
}

// in place: gelu(v), the erf form 0.5 v (1 + erf(v / sqrt 2)) or (tanh_form) 0.5 v (1 + tanh(sqrt(2/pi) (v + 0.044715 v^3)))
template <typename T>
__global__ void gelu_kernel(T* __restrict__ h, int tanh_form, size_t n) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float v = dt<T>::ld(h, i);
  const float r = tanh_form ? 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)))
                            : 0.5f * v * (1.f + erff(v * 0.7071067811865476f));
  dt<T>::st(h, i, r);
}

// Several copies of the residual stream ("hyper-connections"): X [rows][S][dim] fp32.  One launch closes a sublayer and opens
// the next:
//   write   X'[t] = sum_s mix[s][t] X[s] + out[t] * r * ls * y      all S copies at once from the old ones (mix [S][S] indexed
//           [from][to], NULL: every copy keeps itself; y the sublayer's result in the activation dtype, NULL: nothing is added;
//           ls a per-channel scale of y, NULL: none)
//   read    u = sum_t in[t] X'[t] (in NULL: the plain sum);  h = u / sqrt(mean(u^2) + eps) * w      (h NULL: no read)
//   total   (optional) the plain sum of the new copies, fp32 [rows][dim]
// The old copies are read at src + m * src_row + s * src_copy (src_copy 0: every copy starts as the same row, the embedding
// output); when src is X itself and nothing is added or mixed, nothing is written.
template <typename TA, int SMAX>
__global__ void hyper_mix_norm_kernel(const float* src, long long src_row, long long src_copy, float* X, const TA* __restrict__ y,
                                      const float* __restrict__ ls, float r, const float* __restrict__ mix,
                                      const float* __restrict__ w_out, const float* __restrict__ w_in, const float* __restrict__ w,
                                      float eps, void* __restrict__ h, int h_f32, float* __restrict__ total, int S, int dim) {
  extern __shared__ float hyper_us[];            // the row of u
  __shared__ float red[32];
  __shared__ float cm[SMAX * SMAX], co[SMAX], ci[SMAX];
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) cm[i] = mix ? mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) co[i] = w_out ? w_out[i] : 1.f, ci[i] = w_in ? w_in[i] : 1.f;
  __syncthreads();
  const size_t m = blockIdx.x;
  const bool write = y || mix || src != X || src_row != (long long)S * dim || src_copy != dim;
  float ss = 0.f;
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    float xs[SMAX];
#pragma unroll
    for (int s = 0; s < SMAX; ++s) xs[s] = s < S ? src[m * src_row + s * src_copy + i] : 0.f;
    float yv = 0.f;
    if (y) {
      yv = dt<TA>::ld(y, m * dim + i);
      if (ls) yv *= ls[i];
      yv *= r;
    }
    float u = 0.f, tot = 0.f;
#pragma unroll
    for (int t = 0; t < SMAX; ++t) {
      if (t >= S) break;
      float xt = xs[t];
      if (mix) {
        xt = 0.f;
#pragma unroll
        for (int s = 0; s < SMAX; ++s)
          if (s < S) xt = fmaf(cm[s * S + t], xs[s], xt);
      }
      if (y) xt = fmaf(co[t], yv, xt);
      if (write) X[(m * S + t) * dim + i] = xt;
      u = fmaf(ci[t], xt, u);
      tot += xt;
    }
    if (total) total[m * dim + i] = tot;
    hyper_us[i] = u;
    ss += u * u;
  }
  if (!h) return;
  ss = block_sum(ss, red);
  const float k = 1.f / sqrtf(ss / (float)dim + eps);
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    const float n = hyper_us[i] * k * w[i];
    if (h_f32) ((float*)h)[m * dim + i] = n;
    else dt<TA>::st((TA*)h, m * dim + i, n);
  }
}

// out[m][:] = x[m][:] / sqrt(mean(x[m][:]^2) + eps) * w      (rows of x_stride / out_stride elements; w fp32 or NULL)
template <typename T>
__global__ void row_norm_kernel(const T* __restrict__ x, int x_stride, const float* __restrict__ w, float eps, T* __restrict__ out,
                                int out_stride, int dim) {
  __shared__ float red[32];
  const T* xr = x + (size_t)blockIdx.x * x_stride;
  T* orow = out + (size_t)blockIdx.x * out_stride;
  float ss = 0.f;
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    const float v = dt<T>::ld(xr, i);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float k = 1.f / sqrtf(ss / (float)dim + eps);
  for (int i = threadIdx.x; i < dim; i += blockDim.x) dt<T>::st(orow, i, dt<T>::ld(xr, i) * k * (w ? w[i] : 1.f));
}

// out[m][c] = a[m][c] * sigmoid(gate[m][c])     (each with its own row stride; out may be a)
template <typename T>
__global__ void sigmoid_gate_mul_kernel(const T* a, int a_stride, const T* __restrict__ gate, int gate_stride, T* out, int out_stride,
                                        int C, size_t n) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const size_t m = i / C, c = i - m * C;
  const float g = dt<T>::ld(gate, m * gate_stride + c);
  dt<T>::st(out, m * out_stride + c, dt<T>::ld(a, m * a_stride + c) / (1.f + expf(-g)));
}

// in place: cap * tanh(v / cap)
__global__ void tanh_cap_kernel(float* __restrict__ x, float cap, float inv_cap, size_t n) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) x[i] = cap * tanhf(x[i] * inv_cap);
}

}  // namespace llb

extern "C" {

int ll_hyper_mix_norm(const float* src, long long src_row, long long src_copy, float* X, const void* y, const float* ls, float r,
                      const float* mix, const float* w_out, const float* w_in, const float* w, float eps, void* h, int h_f32,
                      float* total, int act_dtype, int rows, int S, int dim, ll_stream stream) {
  LL_CHECK_ARG(src && X && rows >= 0 && S >= 1 && dim > 0 && (!h || w) && (!y || w_out), "bad hyper_mix_norm arguments");
  if (S > 8) {
    set_error("hyper_mix_norm: %d copies of the stream (up to 8)", S);
    return LL_ERR_UNSUPPORTED;
  }
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int threads = dim >= 2048 ? 512 : dim >= 512 ? 256 : 128;
  const size_t smem = (size_t)dim * sizeof(float);
  if (smem > 200 * 1024) {
    set_error("hyper_mix_norm: rows of %d numbers", dim);
    return LL_ERR_UNSUPPORTED;
  }
#define LL_HYPER(TA, SM)                                                                                                            \
  {                                                                                                                                 \
    static bool sized = false;                                                                                                      \
    if (!sized && smem > 48 * 1024) {                                                                                               \
      LL_CUDA(cudaFuncSetAttribute(hyper_mix_norm_kernel<TA, SM>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));        \
      sized = true;                                                                                                                 \
    }                                                                                                                               \
    hyper_mix_norm_kernel<TA, SM><<<rows, threads, smem, st>>>(src, src_row, src_copy, X, (const TA*)y, ls, r, mix, w_out, w_in, w, eps, \
                                                              h, h_f32, total, S, dim);                                             \
  }
#define LL_HYPER_S(TA)                                                                                                              \
  if (S == 1) LL_HYPER(TA, 1) else if (S == 2) LL_HYPER(TA, 2) else if (S <= 4) LL_HYPER(TA, 4) else LL_HYPER(TA, 8)
  if (act_dtype == LL_F32) {
    LL_HYPER_S(float)
  } else if (act_dtype == LL_BF16) {
    LL_HYPER_S(__nv_bfloat16)
  } else {
    set_error("hyper_mix_norm: unsupported dtype %d", act_dtype);
    return LL_ERR_UNSUPPORTED;
  }
#undef LL_HYPER_S
#undef LL_HYPER
  LL_LAUNCH_OK("hyper_mix_norm_kernel");
  return LL_OK;
}

int ll_row_norm(const void* x, int x_stride, const float* w, float eps, void* out, int out_stride, int dtype, int rows, int dim,
                ll_stream stream) {
  LL_CHECK_ARG(x && out && rows >= 0 && dim > 0 && x_stride >= dim && out_stride >= dim, "bad row_norm arguments");
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int threads = dim >= 1024 ? 256 : dim >= 256 ? 128 : 64;
  if (dtype == LL_F32) row_norm_kernel<float><<<rows, threads, 0, st>>>((const float*)x, x_stride, w, eps, (float*)out, out_stride, dim);
  else if (dtype == LL_BF16)
    row_norm_kernel<__nv_bfloat16><<<rows, threads, 0, st>>>((const __nv_bfloat16*)x, x_stride, w, eps, (__nv_bfloat16*)out, out_stride,
                                                            dim);
  else {
    set_error("row_norm: unsupported dtype %d", dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("row_norm_kernel");
  return LL_OK;
}

int ll_sigmoid_gate_mul(const void* a, int a_stride, const void* gate, int gate_stride, void* out, int out_stride, int dtype, int rows,
                        int C, ll_stream stream) {
  LL_CHECK_ARG(a && gate && out && rows >= 0 && C > 0, "bad sigmoid_gate_mul arguments");
  const size_t n = (size_t)rows * C;
  if (n == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const unsigned blocks = (unsigned)((n + 255) / 256);
  if (dtype == LL_F32)
    sigmoid_gate_mul_kernel<float><<<blocks, 256, 0, st>>>((const float*)a, a_stride, (const float*)gate, gate_stride, (float*)out,
                                                          out_stride, C, n);
  else if (dtype == LL_BF16)
    sigmoid_gate_mul_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>((const __nv_bfloat16*)a, a_stride, (const __nv_bfloat16*)gate,
                                                                  gate_stride, (__nv_bfloat16*)out, out_stride, C, n);
  else {
    set_error("sigmoid_gate_mul: unsupported dtype %d", dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("sigmoid_gate_mul_kernel");
  return LL_OK;
}

int ll_tanh_cap(float* x, float cap, size_t n, ll_stream stream) {
  LL_CHECK_ARG(x && cap > 0.f, "bad tanh_cap arguments");
  if (n == 0) return LL_OK;
  tanh_cap_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, cap, 1.f / cap, n);
  LL_LAUNCH_OK("tanh_cap_kernel");
  return LL_OK;
}

int ll_add_norm_pair(float* x, const void* a0, float s0, const void* a1, float s1, const void* a2, float s2, const float* w1,
                     const float* w2, float eps, void* out1, int out1_f32, void* out2, int act_dtype, int rows, int dim,
                     ll_stream stream) {
  LL_CHECK_ARG(x && rows >= 0 && dim > 0 && (!out1 || w1) && (!out2 || w2), "bad add_norm_pair arguments");
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int threads = dim >= 2048 ? 512 : dim >= 512 ? 256 : 128;
  if (act_dtype == LL_F32)
    add_norm_pair_kernel<float><<<rows, threads, 0, st>>>(x, (const float*)a0, s0, (const float*)a1, s1, (const float*)a2, s2, w1, w2,
                                                         eps, out1, out1_f32, (float*)out2, dim);
  else if (act_dtype == LL_BF16)
    add_norm_pair_kernel<__nv_bfloat16><<<rows, threads, 0, st>>>(x, (const __nv_bfloat16*)a0, s0, (const __nv_bfloat16*)a1, s1,
                                                                 (const __nv_bfloat16*)a2, s2, w1, w2, eps, out1, out1_f32,
                                                                 (__nv_bfloat16*)out2, dim);
  else {
    set_error("add_norm_pair: unsupported dtype %d", act_dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("add_norm_pair_kernel");
  return LL_OK;
}

int ll_add_layer_norm(float* x, const void* a, float s, const float* w, const float* b, float eps, void* out, int act_dtype, int rows,
                      int dim, ll_stream stream) {
  LL_CHECK_ARG(x && rows >= 0 && dim > 0 && (!out || (w && b)), "bad add_layer_norm arguments");
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  if (act_dtype == LL_F32) return add_row_norm_launch<float, false>(x, a, s, nullptr, nullptr, w, b, eps, out, rows, dim, st);
  if (act_dtype == LL_BF16) return add_row_norm_launch<__nv_bfloat16, false>(x, a, s, nullptr, nullptr, w, b, eps, out, rows, dim, st);
  set_error("add_layer_norm: unsupported dtype %d", act_dtype);
  return LL_ERR_UNSUPPORTED;
}

int ll_add_rms_norm(float* x, const void* a, float s, const float* a_bias, const float* step, const float* w, float eps, void* out,
                    int act_dtype, int rows, int dim, ll_stream stream) {
  LL_CHECK_ARG(x && rows >= 0 && dim > 0 && (!out || w), "bad add_rms_norm arguments");
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  if (act_dtype == LL_F32) return add_row_norm_launch<float, true>(x, a, s, a_bias, step, w, nullptr, eps, out, rows, dim, st);
  if (act_dtype == LL_BF16) return add_row_norm_launch<__nv_bfloat16, true>(x, a, s, a_bias, step, w, nullptr, eps, out, rows, dim, st);
  set_error("add_rms_norm: unsupported dtype %d", act_dtype);
  return LL_ERR_UNSUPPORTED;
}

int ll_gated_group_norm(const float* y, int y_gs, const float* stab, const void* gate, int gate_stride, const float* w, int w_shared,
                        float eps, int groups, int gate_first, int gate_sigmoid, void* out, int act_dtype, int rows, int C,
                        ll_stream stream) {
  return ll_gated_group_norm_rows(y, y_gs, stab, gate, gate_stride, w, w_shared, eps, groups, gate_first, gate_sigmoid, out, C, act_dtype,
                                  rows, C, stream);
}

int ll_gated_group_norm_rows(const float* y, int y_gs, const float* stab, const void* gate, int gate_stride, const float* w, int w_shared,
                             float eps, int groups, int gate_first, int gate_sigmoid, void* out, int out_stride, int act_dtype, int rows,
                             int C, ll_stream stream) {
  LL_CHECK_ARG(y && gate && w && out && rows >= 0 && C > 0 && groups > 0 && C % groups == 0 && gate_stride >= C && out_stride >= C,
               "bad gated_group_norm arguments");
  if (y_gs == 0) y_gs = C / groups;
  LL_CHECK_ARG(y_gs >= C / groups + (stab ? 1 : 0), "gated_group_norm: a part of y is shorter than the part it norms");
  if (rows == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int gs = C / groups;
  if (gs >= 256 && gs <= 12288 && !stab && y_gs == gs && rows <= 65535) {
    if (act_dtype == LL_F32)
      return gated_group_norm_wide_launch<float>(y, gate, gate_stride, w, w_shared, eps, groups, gate_first, gate_sigmoid, out, out_stride, rows, gs, st);
    if (act_dtype == LL_BF16)
      return gated_group_norm_wide_launch<__nv_bfloat16>(y, gate, gate_stride, w, w_shared, eps, groups, gate_first, gate_sigmoid, out, out_stride,
                                                         rows, gs, st);
    set_error("gated_group_norm: unsupported dtype %d", act_dtype);
    return LL_ERR_UNSUPPORTED;
  }
  const uintptr_t at16 = (uintptr_t)y | (uintptr_t)w, at_act = (uintptr_t)gate | (uintptr_t)out;
  if (!stab && gs <= 256 && ((gs | y_gs | gate_stride | out_stride) & 3) == 0 && (at16 & 15) == 0 &&
      (at_act & (act_dtype == LL_F32 ? 15 : 7)) == 0 && (long long)rows * groups < (1ll << 31)) {
    if (act_dtype == LL_F32)
      return gated_group_norm4_launch<float>(y, y_gs, gate, gate_stride, w, w_shared, eps, groups, gate_first, gate_sigmoid, out, out_stride,
                                             rows, gs, st);
    if (act_dtype == LL_BF16)
      return gated_group_norm4_launch<__nv_bfloat16>(y, y_gs, gate, gate_stride, w, w_shared, eps, groups, gate_first, gate_sigmoid, out,
                                                     out_stride, rows, gs, st);
  }
  const int threads = groups >= 8 ? 256 : groups >= 4 ? 128 : 32 * groups;
  if (act_dtype == LL_F32)
    gated_group_norm_kernel<float><<<rows, threads, 0, st>>>(y, y_gs, stab, (const float*)gate, gate_stride, w, w_shared, eps, groups,
                                                            gate_first, gate_sigmoid, (float*)out, out_stride, C);
  else if (act_dtype == LL_BF16)
    gated_group_norm_kernel<__nv_bfloat16><<<rows, threads, 0, st>>>(y, y_gs, stab, (const __nv_bfloat16*)gate, gate_stride, w, w_shared,
                                                                    eps, groups, gate_first, gate_sigmoid, (__nv_bfloat16*)out,
                                                                    out_stride, C);
  else {
    set_error("gated_group_norm: unsupported dtype %d", act_dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("gated_group_norm_kernel");
  return LL_OK;
}

int ll_relu_squared(void* h, int dtype, size_t n, ll_stream stream) {
  LL_CHECK_ARG(h, "relu_squared: null pointer");
  if (n == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const unsigned blocks = (unsigned)((n + 255) / 256);
  const bool vec = n % 8 == 0 && ((uintptr_t)h & 15) == 0;
  const unsigned blocks8 = (unsigned)((n / 8 + 127) / 128);
  if (dtype == LL_F32 && vec) relu_squared8_kernel<float><<<blocks8, 128, 0, st>>>((float*)h, n / 8);
  else if (dtype == LL_BF16 && vec) relu_squared8_kernel<__nv_bfloat16><<<blocks8, 128, 0, st>>>((__nv_bfloat16*)h, n / 8);
  else if (dtype == LL_F32) relu_squared_kernel<float><<<blocks, 256, 0, st>>>((float*)h, n);
  else if (dtype == LL_BF16) relu_squared_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>((__nv_bfloat16*)h, n);
  else {
    set_error("relu_squared: unsupported dtype %d", dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("relu_squared_kernel");
  return LL_OK;
}

int ll_gelu(void* h, int dtype, int tanh_form, size_t n, ll_stream stream) {
  LL_CHECK_ARG(h, "gelu: null pointer");
  if (n == 0) return LL_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const unsigned blocks = (unsigned)((n + 255) / 256);
  if (dtype == LL_F32) gelu_kernel<float><<<blocks, 256, 0, st>>>((float*)h, tanh_form, n);
  else if (dtype == LL_BF16) gelu_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>((__nv_bfloat16*)h, tanh_form, n);
  else {
    set_error("gelu: unsupported dtype %d", dtype);
    return LL_ERR_UNSUPPORTED;
  }
  LL_LAUNCH_OK("gelu_kernel");
  return LL_OK;
}

}  // extern "C"
