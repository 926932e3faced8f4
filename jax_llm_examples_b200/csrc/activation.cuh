// Pointwise activations by number, shared by the kernels that apply one (bias_act, the streaming product's epilogue).
#pragma once
#include "common.cuh"

enum { ACT_NONE = 0, ACT_RELU2 = 1, ACT_SILU = 2, ACT_GELU_TANH = 3, ACT_GELU = 4, ACT_TANH = 5 };

__device__ __forceinline__ float activate(float z, int act) {
  switch (act) {
    case ACT_RELU2: { const float r = fmaxf(z, 0.f); return r * r; }
    case ACT_SILU: return z / (1.f + expf(-z));
    case ACT_GELU: return 0.5f * z * (1.f + erff(z * 0.7071067811865476f));
    case ACT_TANH: return tanhf(z);
    case ACT_GELU_TANH: return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    default: return z;
  }
}
