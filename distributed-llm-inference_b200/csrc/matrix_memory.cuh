// What the kernels of the matrix memory share: its gates as logarithms, and the divisor of a read-out.
#pragma once
#include "common.cuh"

namespace dli {

__device__ __forceinline__ float memory_in_gate(float z, float cap) { return cap * tanhf(z / cap); }
// logsigmoid(y) = min(y, 0) - log(1 + exp(-|y|)), y = cap tanh(z / cap)
__device__ __forceinline__ float memory_forget_gate(float z, float cap) {
  const float y = cap * tanhf(z / cap);
  return fminf(y, 0.f) - log1pf(expf(-fabsf(y)));
}
__device__ __forceinline__ float memory_divisor(float nq, float m) { return fmaxf(fabsf(nq), expf(-m)) + 1e-6f; }

}  // namespace dli
