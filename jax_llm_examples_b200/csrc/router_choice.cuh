// The choice of experts by a corrected, group-limited router, one warp per token: shared by the router kernels (moe.cu) and
// by the kernel that closes a sublayer and routes in one launch (close_route.cu).
#pragma once
#include "common.cuh"

#define ROUTER_MAX_E 256
#define ROUTER_MAX_K 16
#define ROUTER_MAX_GROUPS 64

// What the choice needs beyond the scores, for the corrected forms: weight_form 2, s = softmax(z) over all E outputs, and
// weight_form 3, s = sigmoid(z).  The choice is made on s + correction, and only among the `keep` best of `groups`
// equal groups of neighbouring outputs (a group's score: the sum of its `group_top` largest s + correction, one or two;
// the others count as -inf, not 0: corrections may be negative); the weights are the chosen s, with `normalize` divided
// by their sum (+ 1e-20), times `scale`.
struct RouterChoice {
  const float* correction;  // [E] or null
  int groups, keep;         // groups <= 1: no limit
  float scale;
  int group_top, normalize;
};

// Called by all 32 lanes of one warp.  `sc` (shared memory, E entries) holds the router's raw scores and is used up.  The k
// largest choice scores in order (the lower index wins a tie) go to idx, their weights to w.  A lane keeps the shares of
// outputs lane, lane + 32, ...; the groups' scores are made a group per lane, and a group is kept when fewer than `keep`
// groups are better.
__device__ __forceinline__ void choose_experts_corrected(float* sc, int E, int k, int* idx, float* w, int weight_form, const RouterChoice& ch) {
  constexpr int PER = ROUTER_MAX_E / 32;
  const int lane = threadIdx.x & 31;
  float s[PER], c[PER];
  float m = -INFINITY, sum = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < E ? sc[e] : -INFINITY;
    m = fmaxf(m, s[i]);
  }
  if (weight_form == 2) m = warp_max(m);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i;
    if (e < E) {
      s[i] = weight_form == 3 ? 1.f / (1.f + expf(-s[i])) : expf(s[i] - m);
      sum += s[i];
    }
  }
  if (weight_form == 2) {
    sum = warp_sum(sum);
#pragma unroll
    for (int i = 0; i < PER; ++i) s[i] = s[i] / sum;
  }
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i;
    c[i] = e < E ? s[i] + (ch.correction ? ch.correction[e] : 0.f) : NAN;  // NaN: never chosen
  }
  if (ch.groups > 1 && ch.keep < ch.groups) {
    const int per = E / ch.groups;
    __syncwarp();  // every lane has read its raw scores
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (lane + 32 * i < E) sc[lane + 32 * i] = c[i];
    __syncwarp();
    float gv[ROUTER_MAX_GROUPS / 32];  // the scores of groups lane and lane + 32
#pragma unroll
    for (int u = 0; u < ROUTER_MAX_GROUPS / 32; ++u) {
      const int g = lane + 32 * u;
      float first = -INFINITY, second = -INFINITY;
      if (g < ch.groups)
        for (int e = g * per; e < (g + 1) * per; ++e) {
          const float v = sc[e];
          second = fmaxf(second, fminf(first, v));
          first = fmaxf(first, v);
        }
      gv[u] = ch.group_top == 2 && per > 1 ? first + second : first;
    }
    __syncwarp();
    unsigned long long allowed = 0ull;  // bit g: group g may be chosen from
#pragma unroll
    for (int u = 0; u < ROUTER_MAX_GROUPS / 32; ++u) {
      const int g = lane + 32 * u;
      int better = 0;
      for (int o = 0; o < ch.groups; ++o) {
        const float a = __shfl_sync(0xffffffffu, gv[0], o & 31), b = __shfl_sync(0xffffffffu, gv[1], o & 31);
        const float ov = o < 32 ? a : b;
        better += ov > gv[u] || (ov == gv[u] && o < g);
      }
      allowed |= (unsigned long long)__ballot_sync(0xffffffffu, g < ch.groups && better < ch.keep) << (32 * u);
    }
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (lane + 32 * i < E && !((allowed >> ((lane + 32 * i) / per)) & 1ull)) c[i] = NAN;
  }
  float total = 0.f;
  float w_mine = 0.f;  // lane j keeps the j-th choice
  int idx_mine = lane;  // nothing left to choose (NaNs everywhere): still a valid index, with no weight
  for (int j = 0; j < k; ++j) {
    int best = -1;
    float bv = 0.f, bs = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (c[i] == c[i] && (best < 0 || c[i] > bv)) {
        best = lane + 32 * i;
        bv = c[i];
        bs = s[i];
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const int ob = __shfl_xor_sync(0xffffffffu, best, o);
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o), os = __shfl_xor_sync(0xffffffffu, bs, o);
      if (ob >= 0 && (best < 0 || ov > bv || (ov == bv && ob < best))) {
        best = ob;
        bv = ov;
        bs = os;
      }
    }
    if (best < 0) break;  // the same for all lanes
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (lane + 32 * i == best) c[i] = NAN;
    if (lane == j) {
      idx_mine = best;
      w_mine = bs;
    }
    total += bs;
  }
  if (lane < k) {
    idx[lane] = idx_mine;
    w[lane] = (ch.normalize ? w_mine / (total + 1e-20f) : w_mine) * ch.scale;
  }
}
