// Soft-capped attention scores: s <- cap * tanh(s / cap).  tanh in float32 without the library's function in the inner
// loop of the tensor-core kernels.
//
// |x| <= 1: x * p(x^2), p the polynomial of degree 5 with the smallest largest relative error against tanh(x) / x on
// [0, 1] (fitted by iteratively reweighted least squares in a Chebyshev basis; 5.9e-7 before rounding).
// |x| > 1: 1 - 2 / (2^(2 x log2 e) + 1), from the definition; there the subtraction cancels nothing.
#pragma once
#include "common.cuh"

#define CAP_C0 0.99999941f
#define CAP_C1 -0.33329042f
#define CAP_C2 0.13281433f
#define CAP_C3 -0.05160566f
#define CAP_C4 0.01674311f
#define CAP_C5 -0.00306706f

__device__ __forceinline__ float cap_tanh_small(float x) {
  const float u = x * x;
  float p = fmaf(CAP_C5, u, CAP_C4);
  p = fmaf(p, u, CAP_C3);
  p = fmaf(p, u, CAP_C2);
  p = fmaf(p, u, CAP_C1);
  p = fmaf(p, u, CAP_C0);
  return p * x;
}

__device__ __forceinline__ float cap_tanh_large(float x) {
  const float e = exp2f(2.8853900817779268f * fabsf(x));  // 2^(2 |x| log2 e): infinite for large |x|, and tanh is 1
  return copysignf(1.f - __fdividef(2.f, fminf(e, 1.0e30f) + 1.f), x);
}

__device__ __forceinline__ float cap_tanh(float x) { return fabsf(x) <= 1.f ? cap_tanh_small(x) : cap_tanh_large(x); }
