// Gated activations of the GEMM epilogues.  act 1: silu(gate) * up, both rounded to bf16 first (as a GEMM that stores them
// would).  act 2: g * sigmoid(1.702 g) * (u + 1) with g = min(gate, limit), u = up clamped to +-limit, in fp32.  act 3 has no gate: the
// squared ReLU of every column.
#pragma once
#include "blaze/sm100.cuh"

namespace blz {

__device__ __forceinline__ float clamped_glu(float gate, float up, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}
// the same with the fast exponential, for results that are rounded to bf16
__device__ __forceinline__ float clamped_glu_fast(float gate, float up, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return __fdividef(g, 1.f + __expf(-1.702f * g)) * (u + 1.f);
}

__device__ __forceinline__ float squared_relu(float x) { const float y = fmaxf(x, 0.f); return y * y; }

}  // namespace blz
