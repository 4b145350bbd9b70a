// What the two forms of the gated delta rule (delta_rule.cu, delta_chunk.cu) share.
#pragma once
#include "common.cuh"

namespace llb {

// log of the decay, -exp(a_log) * softplus(raw + dt_bias)
__device__ __forceinline__ float delta_log_decay(float raw, float dt_bias, float a_log) {
  const float z = raw + dt_bias;
  return -expf(a_log) * (z > 20.f ? z : log1pf(expf(z)));
}
// write strength, sigmoid(raw)
__device__ __forceinline__ float delta_strength(float raw) { return 1.f / (1.f + expf(-raw)); }

}  // namespace llb
