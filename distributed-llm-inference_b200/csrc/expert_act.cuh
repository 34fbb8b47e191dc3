// Activations of a routed mixture's experts, shared by the kernels for few and for many tokens.
#pragma once
#include "common.cuh"

namespace dli {

// of the gate of a gated expert: 0 silu, 1 gelu with the tanh approximation, 2 x sigmoid(1.702 x)
__device__ __forceinline__ float glu_act(float g, int act) {
  if (act == 1) return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
  if (act == 2) return g / (1.f + expf(-1.702f * g));
  return g / (1.f + expf(-g));
}

// of an expert without a gate: 0 the square of relu, 1 gelu with the tanh approximation, 2 silu
__device__ __forceinline__ float plain_act(float v, int act) {
  if (act == 1) return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
  if (act == 2) return v / (1.f + expf(-v));
  const float r = fmaxf(v, 0.f);
  return r * r;
}

}  // namespace dli
