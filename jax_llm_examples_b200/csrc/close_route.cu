// The kernel between a mixer and a routed feed-forward of a block that norms its sublayers' outputs, for the few rows of a
// decode step:
//
//   x += mult * post_w * rms_norm(delta)      (the mixer's output, closed; split-K partials or gathered rows, delta_rows.cuh)
//   out = x in the activations' type          (what a shared expert would read; may be missing)
//   the corrected, group-limited router on x in 32-bit (router_choice.cuh), the step's (token, choice) pairs sorted by expert
//   (expert_sort.cuh), and every token's row copied to its places in expert order
//
// which is group_norm + router + expert_sort + permute_scale in one launch.  ONE cluster of CLOSE_BLOCKS blocks: block b takes rows
// b, b + CLOSE_BLOCKS, ...; a row stays in its block's shared memory from the closing norm to the gather.  The blocks' choices
// meet through distributed shared memory; every block then sorts all pairs itself (there are few) and copies its own rows;
// block 0 writes what the grouped products read (offsets, tile list) and the pairs' order.
#include <cooperative_groups.h>

#include "common.cuh"
#include "delta_rows.cuh"
#include "expert_sort.cuh"
#include "router_choice.cuh"

#define CLOSE_BLOCKS 8
#define CLOSE_THREADS 1024
#define CLOSE_MAX_ROWS 16
#define CLOSE_MAX_PAIRS 256

struct CloseRouteArgs {
  float* x;
  DeltaRows delta;
  const float* post_w;
  float mult, eps;
  void* out;               // [N, D] in the activations' type, or null
  const float* w_router;   // [E, D]
  const float* bias;       // [E] or null
  int* topk_idx;
  float* topk_w;
  int* offsets;
  int* sorted_pair;
  int* sorted_pos;
  int* tile_list;
  int* n_tiles;
  void* a_sorted;          // [N * k, D]
  int* status;
  RouterChoice choice;
  int weight_form, N, D, E, k, tile_rows;
};

template <typename T> __device__ __forceinline__ void store_row4(T* p, float4 v);
template <> __device__ __forceinline__ void store_row4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store_row4<bf16>(bf16* p, float4 v) {
  uint2 o;
  *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = o;
}

template <typename TO>
__global__ void __launch_bounds__(CLOSE_THREADS, 1) close_route_kernel(const CloseRouteArgs A) {
  JLX_TL(TL_NORM_ROUTER);
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  extern __shared__ __align__(16) float rows_buf[];        // this block's rows: [rows][D]
  __shared__ float scratch[33];
  __shared__ float scores[ROUTER_MAX_E];
  __shared__ int my_choice[CLOSE_MAX_ROWS / CLOSE_BLOCKS][ROUTER_MAX_K];
  __shared__ float my_weight[ROUTER_MAX_K];
  __shared__ int choice[CLOSE_MAX_PAIRS], place[CLOSE_MAX_PAIRS];
  __shared__ int counts[ROUTER_MAX_E + 1];
  const int rank = (int)cluster.block_rank(), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int NW = CLOSE_THREADS / 32;
  const int D4 = A.D >> 2;
  // the weights have left L2 since the layer before: asked back while the predecessor still runs, a share per block
  pdl_launch_dependents();
  {
    const size_t total = (size_t)A.E * A.D * 4, part = (total / CLOSE_BLOCKS + 127) & ~(size_t)127, at = part * rank;
    if (at < total) l2_prefetch_block(reinterpret_cast<const char*>(A.w_router) + at, part < total - at ? part : total - at);
    if (rank == 0) l2_prefetch_block(A.post_w, (size_t)A.D * 4);
  }
  pdl_wait();
  for (int n = rank, u = 0; n < A.N; n += CLOSE_BLOCKS, ++u) {
    float4* row4 = reinterpret_cast<float4*>(rows_buf + (size_t)u * A.D);
    float4* x4 = reinterpret_cast<float4*>(A.x + (size_t)n * A.D);
    float ss = 0.f;
    for (int d = threadIdx.x; d < D4; d += CLOSE_THREADS) {
      const float4 v = delta_at4(A.delta, n, A.D, 4 * d);
      row4[d] = v;
      ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
    const float rms = sqrtf(block_sum(ss, scratch) / (float)A.D + A.eps);
    for (int d = threadIdx.x; d < D4; d += CLOSE_THREADS) {  // (a thread's own entries)
      const float4 v = row4[d], g = reinterpret_cast<const float4*>(A.post_w)[d], xo = x4[d];
      float4 s;
      s.x = fmaf(A.mult, v.x / rms * g.x, xo.x);
      s.y = fmaf(A.mult, v.y / rms * g.y, xo.y);
      s.z = fmaf(A.mult, v.z / rms * g.z, xo.z);
      s.w = fmaf(A.mult, v.w / rms * g.w, xo.w);
      row4[d] = s;
      x4[d] = s;
      if (A.out) store_row4<TO>((TO*)A.out + (size_t)n * A.D + 4 * d, s);
    }
    __syncthreads();
    for (int e = warp; e < A.E; e += NW) {
      const float4* wr = reinterpret_cast<const float4*>(A.w_router + (size_t)e * A.D);
      float s4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
      for (int d = lane; d < D4; d += 32) {
        const float4 a = row4[d], b = wr[d];
        s4[0] = fmaf(a.x, b.x, s4[0]); s4[1] = fmaf(a.y, b.y, s4[1]); s4[2] = fmaf(a.z, b.z, s4[2]); s4[3] = fmaf(a.w, b.w, s4[3]);
      }
      const float s = warp_sum((s4[0] + s4[1]) + (s4[2] + s4[3]));
      if (lane == 0) scores[e] = A.bias ? s + A.bias[e] : s;
    }
    __syncthreads();
    if (warp == 0) {
      choose_experts_corrected(scores, A.E, A.k, my_choice[u], my_weight, A.weight_form, A.choice);
      __syncwarp();
      if (lane < A.k) {
        A.topk_idx[(size_t)n * A.k + lane] = my_choice[u][lane];
        A.topk_w[(size_t)n * A.k + lane] = my_weight[lane];
      }
    }
    __syncthreads();  // scores and weights are free for the next row
  }
  cluster.sync();  // every block's choices are in its shared memory
  const int P = A.N * A.k;
  for (int i = threadIdx.x; i < P; i += CLOSE_THREADS) {
    const int n = i / A.k, j = i - n * A.k;
    choice[i] = cluster.map_shared_rank(&my_choice[0][0], n % CLOSE_BLOCKS)[(n / CLOSE_BLOCKS) * ROUTER_MAX_K + j];
  }
  cluster.sync();  // nobody reads another block's memory after this
  // the counting sort, stable in pair order, by every block for itself
  for (int e = warp; e < A.E; e += NW) {
    int c = 0;
    for (int base = 0; base < P; base += 32) c += __popc(__ballot_sync(0xffffffffu, base + lane < P && choice[base + lane] == e));
    if (lane == 0) counts[e] = c;
  }
  __syncthreads();
  if (warp == 0)
    expert_offsets_and_tiles(counts, A.E, P, 0, A.tile_rows, A.offsets, A.tile_list, A.n_tiles, A.status, rank == 0);
  __syncthreads();
  for (int e = warp; e < A.E; e += NW) {
    int at = counts[e];
    for (int base = 0; base < P; base += 32) {
      const int i = base + lane;
      const bool mine = i < P && choice[i] == e;
      const unsigned mask = __ballot_sync(0xffffffffu, mine);
      if (mine) {
        const int dst = at + __popc(mask & ((1u << lane) - 1u));
        place[i] = dst;
        if (rank == 0) {
          A.sorted_pair[dst] = i;
          A.sorted_pos[i] = dst;
        }
      }
      at += __popc(mask);
    }
  }
  __syncthreads();
  for (int n = rank, u = 0; n < A.N; n += CLOSE_BLOCKS, ++u) {
    const float4* row4 = reinterpret_cast<const float4*>(rows_buf + (size_t)u * A.D);
    for (int d = threadIdx.x; d < D4; d += CLOSE_THREADS) {
      const float4 v = row4[d];
      for (int j = 0; j < A.k; ++j) store_row4<TO>((TO*)A.a_sorted + (size_t)place[n * A.k + j] * A.D + 4 * d, v);
    }
  }
}

// Whether a step of N rows can take this kernel.
JLX_API int jlx_close_route_supported(int N, int D, int E, int k) {
  const int per_block = (N + CLOSE_BLOCKS - 1) / CLOSE_BLOCKS;
  return N >= 1 && N <= CLOSE_MAX_ROWS && N * k <= CLOSE_MAX_PAIRS && k >= 1 && k <= ROUTER_MAX_K && k <= E && E <= ROUTER_MAX_E && D % 4 == 0 &&
         (size_t)per_block * D * 4 <= 160 * 1024;
}

// x: float32 [N, D].  delta: as in jlx_group_norm (split-K partials, or an expert layer's rows in expert order with index,
// weights and k).  tile_rows > 0: the row tiles of the grouped products are listed too (see jlx_expert_sort).
JLX_API int jlx_close_route(float* x, const float* delta, int splits, long long split_stride, const int* delta_index,
                            const float* delta_weights, int delta_k, const float* post_w, float mult, float eps, void* out, int dtype,
                            const float* w_router, const float* bias, int weight_form, const float* correction, int groups, int keep,
                            int group_top, int normalize, float scale, int* topk_idx, float* topk_w, int* offsets, int* sorted_pair,
                            int* sorted_pos, int tile_rows, int* tile_list, int* n_tiles, void* a_sorted, int N, int D, int E, int k,
                            int* status, cudaStream_t stream) {
  JLX_REQUIRE(jlx_close_route_supported(N, D, E, k), "close_route: %d rows of %d, top-%d of %d are not supported", N, D, k, E);
  JLX_REQUIRE(delta && splits >= 1 && post_w && eps > 0.f, "close_route: the sublayer's output, its norm weight and a positive eps are needed");
  JLX_REQUIRE(!delta_index || delta_k >= 1, "close_route: gathered rows need how many a token adds");
  JLX_REQUIRE(weight_form == 2 || weight_form == 3, "close_route: unknown weight form %d", weight_form);
  JLX_REQUIRE(groups >= 1 && groups <= ROUTER_MAX_GROUPS && E % groups == 0 && keep >= 1 && keep <= groups && (group_top == 1 || group_top == 2),
              "close_route: %d groups (keep %d, top %d) of %d outputs", groups, keep, group_top, E);
  JLX_REQUIRE(topk_idx && topk_w && offsets && sorted_pair && sorted_pos && a_sorted && status && (tile_rows == 0 || (tile_list && n_tiles)),
              "close_route: incomplete outputs");
  JLX_REQUIRE((((uintptr_t)x | (uintptr_t)delta | (uintptr_t)post_w | (uintptr_t)out | (uintptr_t)w_router | (uintptr_t)a_sorted) & 15) == 0 &&
                  (split_stride & 3) == 0, "close_route: tensors must be 16-byte aligned");
  CloseRouteArgs A;
  A.x = x; A.delta = DeltaRows{delta, split_stride, delta_index, delta_weights, splits, delta_k};
  A.post_w = post_w; A.mult = mult; A.eps = eps; A.out = out; A.w_router = w_router; A.bias = bias; A.topk_idx = topk_idx; A.topk_w = topk_w;
  A.offsets = offsets; A.sorted_pair = sorted_pair; A.sorted_pos = sorted_pos; A.tile_list = tile_list; A.n_tiles = n_tiles;
  A.a_sorted = a_sorted; A.status = status; A.choice = RouterChoice{correction, groups, keep, scale, group_top, normalize};
  A.weight_form = weight_form; A.N = N; A.D = D; A.E = E; A.k = k; A.tile_rows = tile_rows;
  const size_t smem = (size_t)((N + CLOSE_BLOCKS - 1) / CLOSE_BLOCKS) * D * 4;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(CLOSE_BLOCKS);
  cfg.blockDim = dim3(CLOSE_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = CLOSE_BLOCKS;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  JLX_DISPATCH_DTYPE(dtype, TO, {
    if (smem > 40 * 1024)
      JLX_CUDA(cudaFuncSetAttribute(close_route_kernel<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    JLX_CUDA(cudaLaunchKernelEx(&cfg, close_route_kernel<TO>, A));
  });
  JLX_LAUNCH_CHECK("close_route");
  return 0;
}
