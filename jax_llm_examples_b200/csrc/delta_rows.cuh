// What a norm kernel adds to the residual rows before it norms: shared by the kernels that close a sublayer.
#pragma once
#include "common.cuh"

// Where a row's delta lies.  Without `index`: row r of `delta`.  With it, the delta is an expert layer's output still in
// expert order: the sum over j < k of weights[r k + j] (null: 1) times row index[r k + j], j ascending.  In both cases
// `splits` partials of a row are added first, ascending.
struct DeltaRows {
  const float* p;
  long long split_stride;
  const int* index;
  const float* weights;
  int splits, k;
};

__device__ __forceinline__ float delta_at(const DeltaRows& t, size_t r, int D, int d) {
  if (!t.index) {
    float s = 0.f;
    for (int z = 0; z < t.splits; ++z) s += t.p[(size_t)z * t.split_stride + r * D + d];
    return s;
  }
  float s = 0.f;
  for (int j = 0; j < t.k; ++j) {
    const float* p = t.p + (size_t)t.index[r * t.k + j] * D + d;
    float e = 0.f;
    for (int z = 0; z < t.splits; ++z) e += p[(size_t)z * t.split_stride];
    s = fmaf(t.weights ? t.weights[r * t.k + j] : 1.f, e, s);
  }
  return s;
}

__device__ __forceinline__ float4 delta_at4(const DeltaRows& t, size_t r, int D, int d) {  // entries d .. d + 3
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (!t.index) {
    for (int z = 0; z < t.splits; ++z) {
      const float4 v = *reinterpret_cast<const float4*>(t.p + (size_t)z * t.split_stride + r * D + d);
      s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
    }
    return s;
  }
  for (int j = 0; j < t.k; ++j) {
    const float* p = t.p + (size_t)t.index[r * t.k + j] * D + d;
    float4 e = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int z = 0; z < t.splits; ++z) {
      const float4 v = *reinterpret_cast<const float4*>(p + (size_t)z * t.split_stride);
      e.x += v.x; e.y += v.y; e.z += v.z; e.w += v.w;
    }
    const float w = t.weights ? t.weights[r * t.k + j] : 1.f;
    s.x = fmaf(w, e.x, s.x); s.y = fmaf(w, e.y, s.y); s.z = fmaf(w, e.z, s.z); s.w = fmaf(w, e.w, s.w);
  }
  return s;
}
