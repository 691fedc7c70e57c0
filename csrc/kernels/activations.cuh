// Elementwise activations by code (the table ACTIVATIONS of nkipy_b200/ops/mixers.py).
#pragma once
#include "proj_src.cuh"

namespace nkb {
enum { ACT_SILU = 0, ACT_GELU_TANH = 1, ACT_RELU2 = 2, ACT_TANH = 3, ACT_SIGMOID = 4, ACT_NONE = 5,
       ACT_CLAMPED = 6 /* of a pair: gated_residual.cu */, ACT_XIELU = 7 /* with two parameters: xielu */, ACT_COUNT = 8 };

// GELU in its tanh form is written with the exponential: (1 + tanh u) / 2 = 1 / (1 + exp(-2 u))
__device__ __forceinline__ float apply_act(float z, int kind) {
  switch (kind) {
    case ACT_SILU: return z / (1.f + expf(-z));
    case ACT_GELU_TANH: return z / (1.f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
    case ACT_RELU2: { const float r = fmaxf(z, 0.f); return r * r; }
    case ACT_TANH: return tanhf(z);
    case ACT_SIGMOID: return 1.f / (1.f + expf(-z));
    default: return z;
  }
}

// a z^2 + z / 2 above zero, b (exp(z) - 1 - z) + z / 2 below
__device__ __forceinline__ float xielu(float z, float a, float b) {
  return fmaf(0.5f, z, z > 0.f ? a * z * z : b * (expm1f(z) - z));
}
}  // namespace nkb
