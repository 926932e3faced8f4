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

// The exact gelu for results that are rounded to bfloat16: erf(x) = 1 - (a1 t + ... + a5 t^5) exp(-x^2), t = 1 / (1 + p x),
// x >= 0 (Abramowitz and Stegun, Handbook of Mathematical Functions, 7.1.26: error at most 1.5e-7), odd in x.  A few
// instructions without a branch, for an epilogue in which every thread has hundreds of values.
__device__ __forceinline__ float gelu_for_bf16(float z) {
  const float x = fabsf(z) * 0.7071067811865476f;
  const float t = __fdividef(1.f, fmaf(0.3275911f, x, 1.f));
  float p = fmaf(1.061405429f, t, -1.453152027f);
  p = fmaf(p, t, 1.421413741f);
  p = fmaf(p, t, -0.284496736f);
  p = fmaf(p, t, 0.254829592f);
  const float e = copysignf(1.f - p * t * __expf(-x * x), z);
  return 0.5f * z * (1.f + e);
}
