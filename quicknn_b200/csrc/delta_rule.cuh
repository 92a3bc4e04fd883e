// What the kernels of the gated delta rule share (delta_rule.cu: prompts; delta_step.cu: single tokens).
#pragma once
#include "common.cuh"

namespace qnn {

constexpr int DELTA_MAX_DIM = 256;           // key channels of a head

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float beta_of(float b) { return 1.f / (1.f + expf(-b)); }
__device__ __forceinline__ float decay_of(float a, float rate, float bias) { return expf(-rate * softplus(a + bias)); }

}  // namespace qnn
