// What an expert does to its first product's results, in float32.
#pragma once
#include "common.cuh"

// By kind: 1 gelu (erf form), 2 gelu (tanh form), 3 the square of relu.
__device__ __forceinline__ float plain_activation(float z, int kind) {
  if (kind == 1) return 0.5f * z * (1.0f + erff(z * 0.70710678118654752440f));
  if (kind == 2) return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
  float r = fmaxf(z, 0.f);
  return r * r;
}

// The clamped gated unit: g sigmoid(alpha g) (u + shift), g = min(gate, limit), u = up within +-limit.
__device__ __forceinline__ float gated_unit(float gate, float up, float limit, float alpha, float shift) {
  float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.0f + expf(-alpha * g)) * (u + shift);
}
