// Activations in 32-bit, by the code the products carry (enum Activation).
#pragma once

#include "model.cuh"

namespace lb {

// 0.5 z (1 + tanh(u)) with u = sqrt(2 / pi) (z + 0.044715 z^3), as z / (1 + exp(-2 u)): no cancellation for negative z.
__device__ __forceinline__ float gelu_tanh(float z) {
  const float u2 = 1.5957691216057308f * (z + 0.044715f * z * z * z);
  return z / (1.0f + expf(-u2));
}
__device__ __forceinline__ float activate(float z, int act) {
  if (act == ACT_GELU_ERF) return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f));
  if (act == ACT_GELU_TANH) return gelu_tanh(z);
  return z;
}
__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f32(float z) { return z / (1.0f + expf(-z)); }
// The same with the fast exponential and division (relative error of a few 2^-21), for results that are stored in 16 bits.
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
// ln(1 + exp(z)) without overflow.
__device__ __forceinline__ float softplus_f32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

}  // namespace lb
