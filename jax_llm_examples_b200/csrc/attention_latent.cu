// Attention whose keys and values are up-projections of one cached latent per token, with a rotated key part
// shared by all heads and a per-head sink in the softmax's denominator.  32-bit scores, softmax and sums;
// the cache is 32-bit or bfloat16.
//
// The cache holds, per token, ONE row [c (rank) | k_rot (dr)] (pages: [P, 1, 1, page_size, rank + dr]).  The kernels
// work in the latent space (the up-projections are absorbed into the query and applied to the output by the
// caller, as per-head products):
//   score(t, s, h) = (q_lat[h, t] . c_s + q_rot[t, h] . k_rot_s) * scale          q_lat = W_uk[h]^T q_nope
//   p = exp(score - m) / (sum_s exp(score - m) + exp(sink_h - m))                  causal: s <= t; with a window: t - s < window
//   out_lat[h, t] = sum_s p_s c_s                                                  (value = W_uv[h] out_lat)
//
// latent_kv_prep   from the projected row [dq (q_rank) | dkv (rank) | k_rot (dr)]: weighted RMS norms of the two
//                  latents, the rotation of k_rot, and the page write, in one kernel.
// latent_q_prep    from the projected queries [H, dn + dr]: the unrotated parts head-major (for the per-head
//                  products) and the rotated parts, rotated.
// Rotation: pairs (2i, 2i+1), or with `halves` (i, i + dims/2), i < dims/2, by the angle position * inv_freq[i] in 32-bit;
// entries from `dims` on pass.
#include "common.cuh"
#include "mbarrier.cuh"
#include "mma_sync.cuh"

// The two entries that rotate together as pair i.
__device__ __forceinline__ void rot_pair(int i, int rot_dims, int halves, int* a, int* b) {
  *a = halves ? i : 2 * i;
  *b = halves ? i + (rot_dims >> 1) : 2 * i + 1;
}

__device__ __forceinline__ float row_sum_splits(const float* p, int splits, long long stride) {
  float s = 0.f;
  for (int z = 0; z < splits; ++z) s += p[(size_t)z * stride];
  return s;
}

template <typename TO>
__global__ void latent_kv_prep_kernel(const float* __restrict__ proj, int splits, long long split_stride,
                                      const float* __restrict__ q_norm_w, const float* __restrict__ kv_norm_w, float eps,
                                      const float* __restrict__ inv_freq, int rot_dims, TO* __restrict__ cq, TO* __restrict__ pages,
                                      const int* __restrict__ block_table, int bt_stride, const int* __restrict__ req_of_token,
                                      const int* __restrict__ positions, int q_rank, int rank, int dr, int page_size,
                                      int num_pages, int ld, int halves, int* status) {
  JLX_TL(TL_ROPE);
  pdl_launch_dependents_if_small();
  extern __shared__ float sums[];  // the latent's entries, split-K partials added
  __shared__ float scratch[33];
  const int n = blockIdx.x;
  const float* row = proj + (size_t)n * ld;
  // the step's description is older than the step: the token's place is looked up before the wait for the projected rows
  const int p = positions[n];
  const int page = blockIdx.y ? block_table[(size_t)req_of_token[n] * bt_stride + p / page_size] : 0;
  pdl_wait();
  if (blockIdx.y == 0) {  // the query's latent
    float ss = 0.f;
    for (int i = threadIdx.x; i < q_rank; i += blockDim.x) {
      const float v = row_sum_splits(row + i, splits, split_stride);
      sums[i] = v;
      ss = fmaf(v, v, ss);
    }
    const float rms = sqrtf(block_sum(ss, scratch) / (float)q_rank + eps);
    for (int i = threadIdx.x; i < q_rank; i += blockDim.x) cq[(size_t)n * q_rank + i] = from_f32<TO>(sums[i] / rms * q_norm_w[i]);
    return;
  }
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicOr(status, JLX_STATUS_BAD_PAGE);
    return;
  }
  TO* dst = pages + ((size_t)page * page_size + p % page_size) * (rank + dr);
  // the keys' and values' latent
  float ss = 0.f;
  for (int i = threadIdx.x; i < rank; i += blockDim.x) {
    const float v = row_sum_splits(row + q_rank + i, splits, split_stride);
    sums[i] = v;
    ss = fmaf(v, v, ss);
  }
  // the shared rotated key part
  const float* kr = row + q_rank + rank;
  for (int i = threadIdx.x; i < rot_dims / 2; i += blockDim.x) {
    float sn, cs;
    sincosf((float)p * inv_freq[i], &sn, &cs);
    int ia, ib;
    rot_pair(i, rot_dims, halves, &ia, &ib);
    const float u = row_sum_splits(kr + ia, splits, split_stride), v = row_sum_splits(kr + ib, splits, split_stride);
    dst[rank + ia] = from_f32<TO>(u * cs - v * sn);
    dst[rank + ib] = from_f32<TO>(v * cs + u * sn);
  }
  for (int i = rot_dims + threadIdx.x; i < dr; i += blockDim.x) dst[rank + i] = from_f32<TO>(row_sum_splits(kr + i, splits, split_stride));
  const float rms = sqrtf(block_sum(ss, scratch) / (float)rank + eps);
  for (int i = threadIdx.x; i < rank; i += blockDim.x) dst[i] = from_f32<TO>(sums[i] / rms * kv_norm_w[i]);
}

JLX_API int jlx_latent_kv_prep(const float* proj, int splits, long long split_stride, const float* q_norm_w,
                               const float* kv_norm_w, float eps, const float* inv_freq, int rot_dims, void* cq, void* pages,
                               int dtype, const int* block_table, int bt_stride, const int* req_of_token, const int* positions,
                               int N, int q_rank, int rank, int dr, int page_size, int num_pages, int ld, int halves,
                               int* status, cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && q_rank > 0 && rank > 0 && dr >= 0 && splits >= 1, "latent_kv_prep: bad sizes");
  JLX_REQUIRE(rot_dims >= 0 && rot_dims <= dr && rot_dims % 2 == 0, "latent_kv_prep: %d rotated entries of %d", rot_dims, dr);
  JLX_REQUIRE(eps > 0.f, "latent_kv_prep: eps must be positive");
  JLX_REQUIRE(ld >= q_rank + rank + dr, "latent_kv_prep: rows of %d entries do not hold %d + %d + %d", ld, q_rank, rank, dr);
  const int widest = q_rank > rank ? q_rank : rank;
  JLX_REQUIRE((size_t)widest * 4 <= 48 * 1024, "latent_kv_prep: a latent of %d entries does not fit shared memory", widest);
  if (N == 0) return 0;
  JLX_DISPATCH_DTYPE(dtype, TO, {
    // a block for the query's latent and one for the cached row
    JLX_CUDA(jlx_launch_pdl(latent_kv_prep_kernel<TO>, dim3(N, pages ? 2 : 1), dim3(widest >= 512 ? 256 : 128), sizeof(float) * (size_t)widest, stream, proj, splits, split_stride, q_norm_w, kv_norm_w,
                            eps, inv_freq, rot_dims, (TO*)cq, (TO*)pages, block_table, bt_stride, req_of_token, positions, q_rank,
                            rank, dr, page_size, num_pages, ld, halves, status));
  });
  JLX_LAUNCH_CHECK("latent_kv_prep");
  return 0;
}

// q: float32 [rows, H, dn + dr] (or partials); row b of the outputs is row rows[b] of q (rows null: row b).  q_nope: [H, N, dn]
// in the activation type and q_rot: [N, H, dr] (both or neither); q_full (optional): [H, N, dn + dr], the rotated part rotated
// (for per-head score products).
template <typename TO, typename TR>
__global__ void latent_q_prep_kernel(const float* __restrict__ q, int splits, long long split_stride,
                                     const float* __restrict__ inv_freq, int rot_dims, const int* __restrict__ positions,
                                     TO* __restrict__ q_nope, TR* __restrict__ q_rot, TO* __restrict__ q_full, int N, int H,
                                     int dn, int dr, int halves, const int* __restrict__ rows) {
  JLX_TL(TL_ROPE);
  pdl_launch_dependents_if_small();
  const int b = blockIdx.x, h = blockIdx.y;
  const int n = rows ? rows[b] : b, p = positions[n];
  pdl_wait();
  const float* row = q + ((size_t)n * H + h) * (dn + dr);
  TO* full = q_full ? q_full + ((size_t)h * N + b) * (dn + dr) : nullptr;
  for (int i = threadIdx.x; i < dn; i += blockDim.x) {
    const TO v = from_f32<TO>(row_sum_splits(row + i, splits, split_stride));
    if (q_nope) q_nope[((size_t)h * N + b) * dn + i] = v;
    if (full) full[i] = v;
  }
  const float* qr = row + dn;
  TR* dst = q_rot ? q_rot + ((size_t)b * H + h) * dr : nullptr;
  for (int i = threadIdx.x; i < rot_dims / 2; i += blockDim.x) {
    float sn, cs;
    sincosf((float)p * inv_freq[i], &sn, &cs);
    int ia, ib;
    rot_pair(i, rot_dims, halves, &ia, &ib);
    const float u = row_sum_splits(qr + ia, splits, split_stride), v = row_sum_splits(qr + ib, splits, split_stride);
    const float a = u * cs - v * sn, c = v * cs + u * sn;
    if (dst) { dst[ia] = from_f32<TR>(a); dst[ib] = from_f32<TR>(c); }
    if (full) { full[dn + ia] = from_f32<TO>(a); full[dn + ib] = from_f32<TO>(c); }
  }
  for (int i = rot_dims + threadIdx.x; i < dr; i += blockDim.x) {
    const float v = row_sum_splits(qr + i, splits, split_stride);
    if (dst) dst[i] = from_f32<TR>(v);
    if (full) full[dn + i] = from_f32<TO>(v);
  }
}

JLX_API int jlx_latent_q_prep(const float* q, int splits, long long split_stride, const float* inv_freq, int rot_dims,
                              const int* positions, void* q_nope, int dtype, void* q_rot, int rot_dtype, void* q_full, int N,
                              int H, int dn, int dr, int halves, const int* rows, cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && H > 0 && dn > 0 && dr >= 0 && splits >= 1, "latent_q_prep: bad sizes");
  JLX_REQUIRE(rot_dims >= 0 && rot_dims <= dr && rot_dims % 2 == 0, "latent_q_prep: %d rotated entries of %d", rot_dims, dr);
  JLX_REQUIRE(H <= 65535, "latent_q_prep: too many heads (%d)", H);
  if (N == 0) return 0;
  JLX_DISPATCH_DTYPE(dtype, TO, JLX_DISPATCH_DTYPE(rot_dtype, TR, {
    JLX_CUDA(jlx_launch_pdl(latent_q_prep_kernel<TO, TR>, dim3(N, H), dim3(64), 0, stream, q, splits, split_stride, inv_freq, rot_dims,
                            positions, (TO*)q_nope, (TR*)q_rot, (TO*)q_full, N, H, dn, dr, halves, rows));
  }));
  JLX_LAUNCH_CHECK("latent_q_prep");
  return 0;
}

// ------------------------------------------------------------------------------------------------ attention
// One block serves one query token and up to LAT_WARPS * HPW heads; a warp takes HPW heads, a lane one key of the tile for
// the scores and a slice of the latent for the weighted sums, so that every value read from shared memory serves HPW
// products.  All heads share each tile of keys.  Key tiles are aligned to absolute positions (0, 32, 64, ...), so the
// order of a position's sums depends on the position alone.  The sink opens the running maximum and denominator:
// m = sink, l = exp(sink - m) = 1.
// With a window the walk starts at the tile that holds the first visible key; earlier keys of that tile (whose pages may
// have been given back) are read as zeros and masked.
// With `rows` block b serves token rows[b], whose query and output are row b of theirs (the single decoded tokens of a step that also holds prompt
// portions).  With splits > 1 block z takes the keys [(s0 + z) split_keys, (s0 + z + 1) split_keys), s0 the first visible key's range (a multiple of
// the tile, so tiles stay aligned), and leaves (m, l, unnormalised sums) for the combine kernel; the sink opens split 0.
#define LAT_TILE 32
#define LAT_WARPS 8
#define LAT_MAX_R32 32  // latent size up to 1024
#define LAT_COMBINE_CACHE 512

template <typename TC, typename TO, int HPW, int R32>
__global__ void attention_latent_kernel(const float* __restrict__ q_lat, const float* __restrict__ q_rot,
                                        const TC* __restrict__ pages, const int* __restrict__ block_table, int bt_stride,
                                        const int* __restrict__ req_of_token, const int* __restrict__ positions,
                                        const float* __restrict__ sink, TO* __restrict__ out_lat, int N, int H, int rank,
                                        int dr, int page_size, int num_pages, float scale, const int* __restrict__ rows,
                                        int splits, int split_keys, float* __restrict__ part_acc, float* __restrict__ part_ml,
                                        int ldk, int window, int* status) {
  JLX_TL(TL_ATTN_GENERIC);
  pdl_launch_dependents_if_small();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];
  __shared__ long long row_at[LAT_TILE];  // row number of each key of the tile in the pool, -1: a bad page
  const int dk = rank + dr;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
  float* qs = smem;                     // [nwarp * HPW][dk]
  float* ks = qs + nwarp * HPW * dk;    // [LAT_TILE][ldk]
  const int n = rows ? rows[blockIdx.x] : blockIdx.x;
  const int b = blockIdx.x;  // queries, outputs and partial results are numbered as the blocks are
  const int h0 = (blockIdx.y * nwarp + warp) * HPW;  // the warp's first head
  const int z = blockIdx.z;
  const int p = positions[n], r = req_of_token[n];
  for (int u = 0; u < HPW; ++u) {  // heads beyond H get a zero query: they run along and write nothing
    const int h = h0 + u;
    float* q = qs + (warp * HPW + u) * dk;
    for (int d = lane; d < rank; d += 32) q[d] = h < H ? q_lat[((size_t)h * N + b) * rank + d] : 0.f;
    for (int d = lane; d < dr; d += 32) q[rank + d] = h < H ? q_rot[((size_t)b * H + h) * dr + d] : 0.f;
  }
  const bool has_sink = sink != nullptr && z == 0;
  float m[HPW], l[HPW], acc[HPW][R32];
#pragma unroll
  for (int u = 0; u < HPW; ++u) {
    m[u] = (has_sink && h0 + u < H) ? sink[h0 + u] : -INFINITY;
    l[u] = has_sink ? 1.f : 0.f;
#pragma unroll
    for (int i = 0; i < R32; ++i) acc[u][i] = 0.f;
  }
  const int nd = (rank + 31) >> 5;
  const int lo = window > 0 ? max(0, p - window + 1) : 0;  // the first visible key
  int t_begin = lo / LAT_TILE * LAT_TILE, t_end = p;         // first tile and last key of this block
  if (splits > 1) {
    const int range = (lo / split_keys + z) * split_keys;
    t_begin = max(t_begin, range);
    t_end = min(p, range + split_keys - 1);
  }

  // 16-byte loads of the cached rows where their size and the pool's address allow
  constexpr int VEC = 16 / (int)sizeof(TC);
  const bool wide = (dk % VEC) == 0 && ((uintptr_t)pages & 15) == 0;
  const bool quads = (dk & 3) == 0 && (ldk & 3) == 0;  // scores with 16-byte reads of shared memory
  bool bad_page = false;
  for (int t0 = t_begin; t0 <= t_end; t0 += LAT_TILE) {
    __syncthreads();  // the previous tile is consumed; qs is visible
    const int cnt = min(LAT_TILE, t_end - t0 + 1);
    if (threadIdx.x < cnt) {  // where the tile's rows lie
      const int pos = t0 + threadIdx.x;
      int page = pos >= lo ? block_table[(size_t)r * bt_stride + pos / page_size] : -1;
      if (pos >= lo && (page < 0 || page >= num_pages)) { bad_page = true; page = -1; }
      row_at[threadIdx.x] = page < 0 ? -1 : (long long)page * page_size + pos % page_size;
    }
    __syncthreads();
    if (wide) {
      const int chunks = dk / VEC;
#pragma unroll 4
      for (int idx = threadIdx.x; idx < cnt * chunks; idx += blockDim.x) {
        const int j = idx / chunks, ch = idx - j * chunks;
        const long long at = row_at[j];
        uint4 raw = make_uint4(0u, 0u, 0u, 0u);
        if (at >= 0) raw = *reinterpret_cast<const uint4*>(pages + (size_t)at * dk + ch * VEC);
        const TC* e = reinterpret_cast<const TC*>(&raw);
        float* dst = ks + j * ldk + ch * VEC;
#pragma unroll
        for (int u = 0; u < VEC; ++u) dst[u] = to_f32<TC>(e[u]);
      }
    } else {
      for (int idx = threadIdx.x; idx < cnt * dk; idx += blockDim.x) {
        const int j = idx / dk, d = idx - j * dk;
        const long long at = row_at[j];
        ks[j * ldk + d] = at >= 0 ? to_f32<TC>(pages[(size_t)at * dk + d]) : 0.f;
      }
    }
    __syncthreads();
    float sc[HPW];
#pragma unroll
    for (int u = 0; u < HPW; ++u) sc[u] = -INFINITY;
    const bool seen = lane < cnt && t0 + lane >= lo;
    if (seen) {
      float dot[HPW];
#pragma unroll
      for (int u = 0; u < HPW; ++u) dot[u] = 0.f;
      const float* kr = ks + lane * ldk;
      const float* qr = qs + warp * HPW * dk;
      if (quads) {
        for (int d = 0; d < dk; d += 4) {
          const float4 kv = *reinterpret_cast<const float4*>(kr + d);
#pragma unroll
          for (int u = 0; u < HPW; ++u) {
            const float4 qv = *reinterpret_cast<const float4*>(qr + u * dk + d);
            dot[u] = fmaf(qv.x, kv.x, dot[u]);
            dot[u] = fmaf(qv.y, kv.y, dot[u]);
            dot[u] = fmaf(qv.z, kv.z, dot[u]);
            dot[u] = fmaf(qv.w, kv.w, dot[u]);
          }
        }
      } else {
        for (int d = 0; d < dk; ++d) {
          const float kv = kr[d];
#pragma unroll
          for (int u = 0; u < HPW; ++u) dot[u] = fmaf(qr[u * dk + d], kv, dot[u]);
        }
      }
#pragma unroll
      for (int u = 0; u < HPW; ++u) sc[u] = dot[u] * scale;
    }
    float pj[HPW];
#pragma unroll
    for (int u = 0; u < HPW; ++u) {
      const float m_new = fmaxf(m[u], warp_max(sc[u]));
      const float corr = expf(m[u] - m_new);  // without a sink m is -inf on the first tile: exp(-inf) = 0
      pj[u] = seen ? expf(sc[u] - m_new) : 0.f;
      l[u] = l[u] * corr + warp_sum(pj[u]);
      m[u] = m_new;
#pragma unroll
      for (int i = 0; i < R32; ++i) acc[u][i] *= corr;
    }
    for (int j = 0; j < cnt; ++j) {  // key by key: the lane's entries of the latent are independent sums
      float pv[HPW];
#pragma unroll
      for (int u = 0; u < HPW; ++u) pv[u] = __shfl_sync(0xffffffffu, pj[u], j);
      const float* kj = ks + j * ldk + lane;
#pragma unroll
      for (int i = 0; i < R32; ++i) {
        if (i < nd && lane + 32 * i < rank) {
          const float kv = kj[32 * i];
#pragma unroll
          for (int u = 0; u < HPW; ++u) acc[u][i] = fmaf(pv[u], kv, acc[u][i]);
        }
      }
    }
  }
  if (bad_page) atomicOr(status, JLX_STATUS_BAD_PAGE);
#pragma unroll
  for (int u = 0; u < HPW; ++u) {
    const int h = h0 + u;
    if (h >= H) continue;
    if (splits > 1) {
      const size_t slot = ((size_t)blockIdx.x * H + h) * splits + z;
      if (lane == 0) { part_ml[2 * slot] = m[u]; part_ml[2 * slot + 1] = l[u]; }
#pragma unroll
      for (int i = 0; i < R32; ++i) {
        const int d = lane + 32 * i;
        if (i < nd && d < rank) part_acc[slot * rank + d] = acc[u][i];
      }
    } else {
#pragma unroll
      for (int i = 0; i < R32; ++i) {
        const int d = lane + 32 * i;
        if (i < nd && d < rank) out_lat[((size_t)h * N + b) * rank + d] = from_f32<TO>(acc[u][i] / l[u]);
      }
    }
  }
}

// ---- the same on the tensor cores (mma.sync), for a bfloat16 cache: the decoded tokens of a step
// One block of four warps serves one query token, up to 16 heads (the M rows of the products) and one range of keys.
// Tiles of 32 keys come by cp.async, found row by row through the block table, two in flight; a key's row [c | k_rot] in
// shared memory is padded by 16 bytes so that ldmatrix meets no bank twice.
//   scores   warp w takes keys [8 w, 8 w + 8) of the tile: the whole row against all 16 queries (bfloat16, 32-bit sums)
//   softmax  the scores meet in shared memory; every warp keeps the same running maximum and sum per head (32-bit)
//   values   warp w takes the latent's 16-column pieces w, w + 4, ...: P (bfloat16) times the tile's rows
// When every served token is its request's only one of the step (`single`), everything but its own row is older than the
// step: tiles that end below it are asked for before the wait for the predecessor.  Rows outside [lo, t_end] are zeros in shared memory and masked.
#define LATM_KEYS LAT_TILE
#define LATM_THREADS 128

template <typename TO, int PIECES>
__global__ void __launch_bounds__(LATM_THREADS)
attention_latent_mma_kernel(const bf16* __restrict__ q_lat, const bf16* __restrict__ q_rot, const bf16* __restrict__ pages,
                            const int* __restrict__ block_table, int bt_stride, const int* __restrict__ req_of_token,
                            const int* __restrict__ positions, const float* __restrict__ sink, TO* __restrict__ out_lat, int N,
                            int H, int rank, int dr, int page_size, int num_pages, float scale, const int* __restrict__ rows,
                            int splits, int split_keys, float* __restrict__ part_acc, float* __restrict__ part_ml, int ldk,
                            int window, int single, int* status) {
  JLX_TL(TL_ATTN_GENERIC);
  extern __shared__ __align__(16) uint8_t smem_bytes[];
  __shared__ float sc[2][16][LATM_KEYS + 1];
  const int dk = rank + dr, dkp = (dk + 15) & ~15;  // products take 16 columns at a time: the rest of a row is zero
  bf16* qs = reinterpret_cast<bf16*>(smem_bytes);   // [16][ldk]
  bf16* ks = qs + 16 * ldk;                          // [2][LATM_KEYS][ldk]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int n = rows ? rows[blockIdx.x] : blockIdx.x, h0 = blockIdx.y * 16, z = blockIdx.z;
  const int p = positions[n], r = req_of_token[n];
  const int lo = window > 0 ? max(0, p - window + 1) : 0;
  int t_begin = lo / LATM_KEYS * LATM_KEYS, t_end = p;
  if (splits > 1) {
    const int range = (lo / split_keys + z) * split_keys;
    t_begin = max(t_begin, range);
    t_end = min(p, range + split_keys - 1);
  }
  const int n_tiles = t_begin <= t_end ? (t_end - t_begin) / LATM_KEYS + 1 : 0;
  const int* table = block_table + (size_t)r * bt_stride;
  const int chunks = dk >> 3;  // 16-byte pieces of a row
  bool bad_page = false;
  auto load = [&](int t) {  // a warp copies a row with neighbouring lanes
    bf16* dst = ks + (size_t)(t & 1) * LATM_KEYS * ldk;
    for (int j = warp; j < LATM_KEYS; j += LATM_THREADS / 32) {
      const int pos = t_begin + t * LATM_KEYS + j;
      bool valid = pos >= lo && pos <= t_end;
      const bf16* src = pages;
      if (valid) {
        const int page = table[pos / page_size];
        if (page < 0 || page >= num_pages) { bad_page = true; valid = false; }
        else src = pages + ((size_t)page * page_size + pos % page_size) * dk;
      }
      for (int c = lane; c < chunks; c += 32) cp_async16(smem_u32(dst + (size_t)j * ldk + c * 8), valid ? src + c * 8 : pages, valid);
    }
  };
  // zeros behind every row up to a multiple of 16 columns, once
  if (dkp > dk)
    for (int i = threadIdx.x; i < (2 * LATM_KEYS + 16) * 8; i += LATM_THREADS) qs[(size_t)(i >> 3) * ldk + dk + (i & 7)] = __float2bfloat16_rn(0.f);
  auto old_tile = [&](int t) { return t_begin + (t + 1) * LATM_KEYS <= p; };  // ends below the token's own row
  const bool early0 = single && n_tiles > 0 && old_tile(0), early1 = early0 && n_tiles > 1 && old_tile(1);
  if (early0) { load(0); cp_async_commit(); }
  if (early1) { load(1); cp_async_commit(); }
  pdl_launch_dependents_if_small();
  pdl_wait();
  for (int u = warp; u < 16; u += LATM_THREADS / 32) {  // heads beyond H get a zero query: they run along and write nothing
    const int h = h0 + u;
    const bool valid = h < H;
    const bf16* a = q_lat + ((size_t)(valid ? h : 0) * N + blockIdx.x) * rank;
    const bf16* c = q_rot + ((size_t)blockIdx.x * H + (valid ? h : 0)) * dr;
    const uint32_t dst = smem_u32(qs + (size_t)u * ldk);
    for (int i = lane; i < chunks; i += 32) cp_async16(dst + i * 16, i * 8 < rank ? a + i * 8 : c + (i * 8 - rank), valid);
  }
  if (n_tiles > 0 && !early0) load(0);
  cp_async_commit();
  if (!early1) {
    if (n_tiles > 1) load(1);
    cp_async_commit();  // (maybe empty: the first wait counts groups)
  }
  const int g0 = lane >> 2, g1 = g0 + 8;  // this thread's two heads
  const float sc2 = scale * 1.4426950408889634f;
  const bool has_sink = sink != nullptr && z == 0;
  float m[2], l[2];  // base-2 running maximum and sum
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int h = h0 + (u ? g1 : g0);
    m[u] = has_sink && h < H ? sink[h] * 1.4426950408889634f : -INFINITY;
    l[u] = has_sink ? 1.f : 0.f;
  }
  float o[PIECES][2][4];
#pragma unroll
  for (int i = 0; i < PIECES; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][0][e] = o[i][1][e] = 0.f;

  for (int t = 0; t < n_tiles; ++t) {
    if (t == 0 && !early1) cp_async_wait<1>();  // all but tile 1
    else cp_async_wait<0>();
    __syncthreads();  // tile t has landed for everyone; everyone is done with tile t - 1
    if (t > 0) {
      if (t + 1 < n_tiles) load(t + 1);
      cp_async_commit();
    }
    const bf16* kt = ks + (size_t)(t & 1) * LATM_KEYS * ldk;
    // scores of this warp's 8 keys; two chains of sums
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t qa = smem_u32(qs + (size_t)(lane & 15) * ldk + (lane >> 4) * 8);
    const uint32_t ka = smem_u32(kt + (size_t)(warp * 8 + (lane & 7)) * ldk + (lane >> 3) * 8);
    int d = 0;
    for (; d + 32 <= dkp; d += 32) {
      uint32_t a[4], b[4], c[4];
      ldmatrix_x4(qa + d * 2, a[0], a[1], a[2], a[3]);
      ldmatrix_x4(qa + d * 2 + 32, c[0], c[1], c[2], c[3]);
      ldmatrix_x4(ka + d * 2, b[0], b[1], b[2], b[3]);
      mma_bf16(s0, a, b[0], b[1]);
      mma_bf16(s1, c, b[2], b[3]);
    }
    if (d < dkp) {  // 16 columns are left (lanes 16.. read columns that are in the row's padding or the next row: unused)
      uint32_t a[4], b[4];
      ldmatrix_x4(qa + d * 2, a[0], a[1], a[2], a[3]);
      ldmatrix_x4(smem_u32(kt + (size_t)(warp * 8 + (lane & 7)) * ldk + ((lane >> 3) & 1) * 8) + d * 2, b[0], b[1], b[2], b[3]);
      mma_bf16(s0, a, b[0], b[1]);
    }
    {
      float* w0 = &sc[t & 1][g0][warp * 8 + (lane & 3) * 2];
      float* w1 = &sc[t & 1][g1][warp * 8 + (lane & 3) * 2];
      w0[0] = s0[0] + s1[0]; w0[1] = s0[1] + s1[1];
      w1[0] = s0[2] + s1[2]; w1[1] = s0[3] + s1[3];
    }
    __syncthreads();
    // every warp: the 32 keys' weights of its lanes' two heads, in the layout of the product's A operand
    float pv[2][2][4];  // [16-key step][head][columns 2 (lane & 3) + {0, 1, 8, 9}]
    float mx[2] = {m[0], m[1]};
    const int tile_key = t_begin + t * LATM_KEYS;
#pragma unroll
    for (int st = 0; st < 2; ++st)
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = st * 16 + (lane & 3) * 2 + (e & 1) + (e >> 1) * 8;
          const bool seen = tile_key + j >= lo && tile_key + j <= t_end;
          const float s = seen ? sc[t & 1][u ? g1 : g0][j] * sc2 : -INFINITY;
          pv[st][u][e] = s;
          mx[u] = fmaxf(mx[u], s);
        }
    float corr[2], rs[2] = {0.f, 0.f};
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffffu, mx[u], 1));
      mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffffu, mx[u], 2));  // a tile has a visible key: never -infinity
      corr[u] = exp2f(m[u] - mx[u]);
    }
#pragma unroll
    for (int st = 0; st < 2; ++st)
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          pv[st][u][e] = exp2f(pv[st][u][e] - mx[u]);
          rs[u] += pv[st][u][e];
        }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      rs[u] += __shfl_xor_sync(0xffffffffu, rs[u], 1);
      rs[u] += __shfl_xor_sync(0xffffffffu, rs[u], 2);
      l[u] = l[u] * corr[u] + rs[u];
      m[u] = mx[u];
    }
    uint32_t pa[2][4];
#pragma unroll
    for (int st = 0; st < 2; ++st) {
      pa[st][0] = pack_bf16(pv[st][0][0], pv[st][0][1]);
      pa[st][1] = pack_bf16(pv[st][1][0], pv[st][1][1]);
      pa[st][2] = pack_bf16(pv[st][0][2], pv[st][0][3]);
      pa[st][3] = pack_bf16(pv[st][1][2], pv[st][1][3]);
    }
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
      const int col = (warp + i * 4) * 16;
      if (col >= rank) break;
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        o[i][q][0] *= corr[0]; o[i][q][1] *= corr[0]; o[i][q][2] *= corr[1]; o[i][q][3] *= corr[1];
      }
#pragma unroll
      for (int st = 0; st < 2; ++st) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(smem_u32(kt + (size_t)(st * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * ldk + col + (lane >> 4) * 8), b0, b1, b2, b3);
        mma_bf16(o[i][0], pa[st], b0, b1);
        mma_bf16(o[i][1], pa[st], b2, b3);
      }
    }
  }
  cp_async_wait<0>();
  if (bad_page) atomicOr(status, JLX_STATUS_BAD_PAGE);
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int h = h0 + (u ? g1 : g0);
    if (h >= H) continue;
    const size_t slot = ((size_t)blockIdx.x * H + h) * splits + z;
    if (splits > 1 && warp == 0 && (lane & 3) == 0) {
      part_ml[2 * slot] = m[u] * 0.6931471805599453f;  // the combine kernel works with natural exponentials
      part_ml[2 * slot + 1] = l[u];
    }
    const float inv = 1.f / l[u];
#pragma unroll
    for (int i = 0; i < PIECES; ++i)
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int c = (warp + i * 4) * 16 + q * 8 + (lane & 3) * 2 + e;
          if (c >= rank) continue;
          if (splits > 1) part_acc[slot * rank + c] = o[i][q][u * 2 + e];
          else out_lat[((size_t)h * N + blockIdx.x) * rank + c] = from_f32<TO>(o[i][q][u * 2 + e] * inv);
        }
  }
}

// out = sum_z acc_z exp(m_z - m) / sum_z l_z exp(m_z - m), m = max_z m_z, the splits in ascending order.
template <typename TO>
__global__ void attention_latent_combine_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml,
                                                TO* __restrict__ out_lat, int N, int H, int rank, int splits) {
  JLX_TL(TL_ATTN_COMBINE);
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y;
  const size_t slot0 = ((size_t)b * H + h) * splits;
  __shared__ float ms[LAT_COMBINE_CACHE], wgt[LAT_COMBINE_CACHE];  // the ranges' maxima; their sums, then their shares
  const bool cached = splits <= LAT_COMBINE_CACHE;
  const float2* ml = reinterpret_cast<const float2*>(part_ml) + slot0;
  float m = -INFINITY, l = 0.f;
  if (cached) {
    for (int z = threadIdx.x; z < splits; z += blockDim.x) {
      const float2 v = ml[z];
      ms[z] = v.x;
      wgt[z] = v.y;
    }
    __syncthreads();
    for (int z = 0; z < splits; ++z) m = fmaxf(m, ms[z]);
    for (int z = 0; z < splits; ++z) l += ms[z] > -INFINITY ? wgt[z] * expf(ms[z] - m) : 0.f;
    __syncthreads();
    for (int z = threadIdx.x; z < splits; z += blockDim.x) wgt[z] = ms[z] > -INFINITY ? expf(ms[z] - m) : 0.f;
    __syncthreads();
  } else {
    for (int z = 0; z < splits; ++z) m = fmaxf(m, ml[z].x);
    for (int z = 0; z < splits; ++z) l += ml[z].x > -INFINITY ? ml[z].y * expf(ml[z].x - m) : 0.f;
  }
  for (int d = threadIdx.x; d < rank; d += blockDim.x) {
    float a = 0.f;
#pragma unroll 8
    for (int z = 0; z < splits; ++z) {
      const float w = cached ? wgt[z] : (ml[z].x > -INFINITY ? expf(ml[z].x - m) : 0.f);
      a = fmaf(part_acc[(slot0 + z) * rank + d], w, a);  // (a range without keys left zeros)
    }
    out_lat[((size_t)h * N + b) * rank + d] = from_f32<TO>(a / l);
  }
}

static int latent_combine(const float* part_acc, const float* part_ml, void* out_lat, int out_dtype, int served, int N, int H, int rank,
                          int splits, cudaStream_t stream) {
  if (splits == 1) return 0;
  JLX_DISPATCH_DTYPE(out_dtype, TO, {
    JLX_CUDA(jlx_launch_pdl(attention_latent_combine_kernel<TO>, dim3(served, H), dim3(rank > 256 ? 512 : (rank > 128 ? 256 : 128)), 0, stream, part_acc, part_ml, (TO*)out_lat,
                            N, H, rank, splits));
  });
  JLX_LAUNCH_CHECK("attention_latent_combine");
  return 0;
}

// use_mma: the queries are bfloat16, for the tensor cores (else float32).  single: every served token is its request's only one of
// the step.
// rows / n_rows: serve these token rows only (N = n_rows: queries and outputs in the list's order).  splits > 1: part_acc float32
// [n_rows * H * splits * rank], part_ml float32 [n_rows * H * splits * 2].
JLX_API int jlx_attention_latent(const void* q_lat, const void* q_rot, const void* pages, int cache_dtype,
                                 const int* block_table, int bt_stride, const int* req_of_token, const int* positions,
                                 const float* sink, void* out_lat, int out_dtype, int N, int H, int rank, int dr,
                                 int page_size, int num_pages, float scale, const int* rows, int n_rows, int splits,
                                 int split_keys, float* part_acc, float* part_ml, int window, int use_mma, int single, int* status,
                                 cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && H > 0 && rank > 0 && dr >= 0 && page_size > 0 && num_pages > 0, "attention_latent: bad sizes");
  JLX_REQUIRE(rank <= 32 * LAT_MAX_R32, "attention_latent: latent size %d is above the supported maximum %d", rank, 32 * LAT_MAX_R32);
  JLX_REQUIRE(splits >= 1 && splits <= 65535 && window >= 0, "attention_latent: bad split count %d or window %d", splits, window);
  JLX_REQUIRE(splits == 1 || (split_keys > 0 && split_keys % LAT_TILE == 0 && part_acc && part_ml),
              "attention_latent: splits need a key count that is a multiple of %d, and scratch", LAT_TILE);
  const int served = rows ? n_rows : N;
  if (served == 0) return 0;
  const int dk = rank + dr;
  if (use_mma) {  // on the tensor cores
    JLX_REQUIRE(cache_dtype == JLX_BF16 && rank % 8 == 0 && dr % 8 == 0 && (((uintptr_t)pages | (uintptr_t)q_lat | (uintptr_t)q_rot) & 15) == 0,
                "attention_latent: bfloat16 queries need a bfloat16 cache and sizes that are multiples of 8 (got %d + %d)", rank, dr);
    const int ldm = ((dk + 15) & ~15) + 8;  // rows an odd number of 16-byte pieces apart
    const size_t smem_m = sizeof(bf16) * (size_t)(2 * LATM_KEYS + 16) * ldm;
    const int hb = (H + 15) / 16;
    JLX_REQUIRE(smem_m <= 220 * 1024 && hb <= 65535, "attention_latent: a latent of %d + %d or %d heads are too many", rank, dr, H);
#define LATM_GO(PIECES)                                                                                                        \
  do {                                                                                                                         \
    if (smem_m > 48 * 1024)                                                                                                    \
      JLX_CUDA(cudaFuncSetAttribute(attention_latent_mma_kernel<TO, PIECES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_m)); \
    JLX_CUDA(jlx_launch_pdl(attention_latent_mma_kernel<TO, PIECES>, dim3(served, hb, splits), dim3(LATM_THREADS), smem_m, stream, (const bf16*)q_lat, \
                            (const bf16*)q_rot, (const bf16*)pages, block_table, bt_stride, req_of_token, positions, sink, (TO*)out_lat, N, H, rank, \
                            dr, page_size, num_pages, scale, rows, splits, split_keys, part_acc, part_ml, ldm, window, single, status)); \
  } while (0)
    JLX_DISPATCH_DTYPE(out_dtype, TO, {
      if (rank <= 128) LATM_GO(2);
      else if (rank <= 512) LATM_GO(8);
      else LATM_GO(16);
    });
#undef LATM_GO
    JLX_LAUNCH_CHECK("attention_latent_mma");
    return latent_combine(part_acc, part_ml, out_lat, out_dtype, served, N, H, rank, splits, stream);
  }
  // a key's row in shared memory: padded so that 16-byte reads of a quarter warp's rows fall into different banks
  // (rows a multiple of 4 floats apart with an odd count of 16-byte pieces), else by one float
  const int ldk = (dk & 3) == 0 ? (((dk >> 2) & 1) ? dk : dk + 4) : dk + 1;
  const bool big = rank > 512;             // latents above 512: two heads per warp, else four
  const int hpw = big ? 2 : 4;
  const int groups = (H + hpw - 1) / hpw;  // warps' worth of heads
  int nwarp = groups < LAT_WARPS ? groups : LAT_WARPS;
  auto smem_for = [&](int warps) { return sizeof(float) * ((size_t)warps * hpw * dk + (size_t)LAT_TILE * ldk); };
  while (nwarp > 1 && smem_for(nwarp) > 200 * 1024) nwarp >>= 1;  // fewer heads per block where the rows are long
  const size_t smem = smem_for(nwarp);
  JLX_REQUIRE(smem <= 200 * 1024, "attention_latent: a key tile of %d x %d does not fit into shared memory", LAT_TILE, dk);
  const int hb = (groups + nwarp - 1) / nwarp;
  JLX_REQUIRE(hb <= 65535 && H <= 65535, "attention_latent: too many heads (%d)", H);
#define LAT_GO(HPW, R32)                                                                                                   \
  do {                                                                                                                     \
    if (smem > 48 * 1024)                                                                                                  \
      JLX_CUDA(cudaFuncSetAttribute(attention_latent_kernel<TC, TO, HPW, R32>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                    (int)smem));                                                                           \
    JLX_CUDA(jlx_launch_pdl(attention_latent_kernel<TC, TO, HPW, R32>, dim3(served, hb, splits), dim3(nwarp * 32), smem, stream, \
                            (const float*)q_lat, (const float*)q_rot, (const TC*)pages, block_table, bt_stride, req_of_token, positions, sink, (TO*)out_lat, \
                            N, H, rank, dr, page_size, num_pages, scale, rows, splits, split_keys, part_acc, part_ml, ldk,  \
                            window, status));                                                                                      \
  } while (0)
  JLX_DISPATCH_DTYPE(cache_dtype, TC, JLX_DISPATCH_DTYPE(out_dtype, TO, {
    if (big) LAT_GO(2, 32);
    else LAT_GO(4, 16);
  }));
#undef LAT_GO
  JLX_LAUNCH_CHECK("attention_latent");
  return latent_combine(part_acc, part_ml, out_lat, out_dtype, served, N, H, rank, splits, stream);
}

// ------------------------------------------------------------------------------------------------ prompt portions
// For a prompt portion the scores and the weighted sums are per-head matrix products on the tensor cores (the caller's,
// from the library), around three kernels of this file: the request's cached rows gathered into two dense matrices,
// the keys put together per head, and the softmax with its causal edge and its sink.

// c[t, :] = the first `rank` entries of the cache row of position first + t, kr[t, :] = its last dr, t < L, for the
// request of one block-table row.
template <typename T>
__global__ void latent_gather_kernel(const T* __restrict__ pages, const int* __restrict__ bt_row, T* __restrict__ c,
                                     T* __restrict__ kr, int first, int rank, int dr, int page_size, int num_pages,
                                     int* status) {
  JLX_TL(TL_OTHER);
  const int t = blockIdx.x, pos = first + t;
  const int page = bt_row[pos / page_size];
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicOr(status, JLX_STATUS_BAD_PAGE);
    return;
  }
  const T* src = pages + ((size_t)page * page_size + pos % page_size) * (rank + dr);
  for (int i = threadIdx.x; i < rank; i += blockDim.x) c[(size_t)t * rank + i] = src[i];
  for (int i = threadIdx.x; i < dr; i += blockDim.x) kr[(size_t)t * dr + i] = src[rank + i];
}

JLX_API int jlx_latent_gather(const void* pages, int dtype, const int* bt_row, void* c, void* kr, int first, int L, int rank, int dr,
                              int page_size, int num_pages, int* status, cudaStream_t stream) {
  JLX_REQUIRE(L >= 0 && first >= 0 && rank > 0 && dr >= 0 && page_size > 0, "latent_gather: bad sizes");
  if (L == 0) return 0;
  JLX_DISPATCH_DTYPE(dtype, T, {
    latent_gather_kernel<T><<<L, 128, 0, stream>>>((const T*)pages, bt_row, (T*)c, (T*)kr, first, rank, dr, page_size, num_pages, status);
  });
  JLX_LAUNCH_CHECK("latent_gather");
  return 0;
}

// k[h, t, :] = [kv_up[t, h * dn .. (h + 1) * dn) | kr[t, :]]: every head's key with the shared rotated part appended.
template <typename T>
__global__ void latent_key_assemble_kernel(const T* __restrict__ kv_up, long long ld_up, const T* __restrict__ kr,
                                           T* __restrict__ k, int L, int H, int dn, int dr) {
  JLX_TL(TL_OTHER);
  const int t = blockIdx.x, d = dn + dr;
  for (int i = threadIdx.x; i < H * d; i += blockDim.x) {
    const int h = i / d, e = i - h * d;
    k[((size_t)h * L + t) * d + e] = e < dn ? kv_up[(size_t)t * ld_up + h * dn + e] : kr[(size_t)t * dr + (e - dn)];
  }
}

JLX_API int jlx_latent_key_assemble(const void* kv_up, long long ld_up, const void* kr, void* k, int dtype, int L, int H,
                                    int dn, int dr, cudaStream_t stream) {
  JLX_REQUIRE(L >= 0 && H > 0 && dn > 0 && dr >= 0 && ld_up >= (long long)H * dn, "latent_key_assemble: bad sizes");
  if (L == 0) return 0;
  JLX_DISPATCH_DTYPE(dtype, T, {
    latent_key_assemble_kernel<T><<<L, 256, 0, stream>>>((const T*)kv_up, ld_up, (const T*)kr, (T*)k, L, H, dn, dr);
  });
  JLX_LAUNCH_CHECK("latent_key_assemble");
  return 0;
}

// p[h, i, j] = exp(scale * s[h, i, j] - m) / (sum over visible j + exp(sink_h - m)) for visible j, else 0.  Column j is the
// key at position k_start + j, row i the query at q_start + i: it sees keys up to itself, with a window only the last
// `window` of them.
// s: float32 [H, T, L]; p: [H, T, L] in the activations' type.  One block per (query row, head); 32-bit throughout.
// With `staged` the visible part of the row is read once into shared memory (L floats) and the three passes run there.
template <typename TO>
__global__ void causal_sink_softmax_kernel(const float* __restrict__ s, const float* __restrict__ sink, float scale,
                                           int q_start, int k_start, int window, TO* __restrict__ p, int T, int L,
                                           int staged) {
  JLX_TL(TL_OTHER);
  extern __shared__ __align__(16) float stage[];
  __shared__ float scratch[33];
  const int i = blockIdx.x, h = blockIdx.y;
  const float* row = s + ((size_t)h * T + i) * L;
  TO* out = p + ((size_t)h * T + i) * L;
  const int own = q_start + i - k_start;                             // the query's own column
  const int visible = min(L, own + 1);                               // columns [first, visible) are seen
  const int first = window > 0 ? max(0, own - window + 1) : 0;
  float m = sink ? sink[h] : -INFINITY;
  if (staged) {
    if ((L & 3) == 0) {  // rows start on 16-byte boundaries
      for (int j = (first & ~3) + threadIdx.x * 4; j < visible; j += blockDim.x * 4) {
        float4 v = *reinterpret_cast<const float4*>(row + j);
        v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
        *reinterpret_cast<float4*>(stage + j) = v;
        if (j >= first) m = fmaxf(m, v.x);
        if (j + 1 >= first && j + 1 < visible) m = fmaxf(m, v.y);
        if (j + 2 >= first && j + 2 < visible) m = fmaxf(m, v.z);
        if (j + 3 >= first && j + 3 < visible) m = fmaxf(m, v.w);
      }
    } else {
      for (int j = first + threadIdx.x; j < visible; j += blockDim.x) { stage[j] = row[j] * scale; m = fmaxf(m, stage[j]); }
    }
    row = stage;
    scale = 1.f;
  } else {
    for (int j = first + threadIdx.x; j < visible; j += blockDim.x) m = fmaxf(m, row[j] * scale);
  }
  // the block's maximum: warp maxima, then every thread takes the largest
  m = warp_max(m);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = m;
  __syncthreads();
  m = scratch[0];
  for (int w = 1; w < (blockDim.x >> 5); ++w) m = fmaxf(m, scratch[w]);
  float l = 0.f;
  for (int j = first + threadIdx.x; j < visible; j += blockDim.x) l += expf(row[j] * scale - m);
  l = block_sum(l, scratch) + (sink ? expf(sink[h] - m) : 0.f);
  for (int j = threadIdx.x; j < L; j += blockDim.x) out[j] = from_f32<TO>(j >= first && j < visible ? expf(row[j] * scale - m) / l : 0.f);
}

JLX_API int jlx_causal_sink_softmax(const float* s, const float* sink, float scale, int q_start, int k_start, int window, void* p,
                                    int dtype, int H, int T, int L, cudaStream_t stream) {
  JLX_REQUIRE(H > 0 && T >= 0 && L > 0 && q_start >= 0 && k_start >= 0 && k_start <= q_start && window >= 0 && H <= 65535, "causal_sink_softmax: bad sizes");
  if (T == 0) return 0;
  const int staged = (size_t)L * 4 <= 160 * 1024;
  const size_t smem = staged ? (size_t)(L + 4) * 4 : 0;
  JLX_DISPATCH_DTYPE(dtype, TO, {
    if (smem > 48 * 1024)
      JLX_CUDA(cudaFuncSetAttribute(causal_sink_softmax_kernel<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    causal_sink_softmax_kernel<TO><<<dim3(T, H), 256, smem, stream>>>(s, sink, scale, q_start, k_start, window, (TO*)p, T, L, staged);
  });
  JLX_LAUNCH_CHECK("causal_sink_softmax");
  return 0;
}

// [H, N, d] -> [N, H * d]: the per-head products' rows back into token rows, with `gate` (float32 rows, possibly split-K
// partials) through a gate per token and head: out[n, h d + c] = sigmoid(gate[n, h]) * in[h, n, c].  With `rows` row b of
// the input belongs to token rows[b].
struct GateRowsView {
  const float* p;
  long long split_stride;
  long long ld;
  int splits;
  int pad_;
};

template <typename T>
__global__ void heads_to_rows_kernel(const T* __restrict__ in, T* __restrict__ out, int N, int H, int d, GateRowsView gate,
                                     const int* __restrict__ rows) {
  JLX_TL(TL_OTHER);
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int b = blockIdx.x, n = rows ? rows[b] : b;
  constexpr int VEC = 16 / (int)sizeof(T);
  if (d % VEC == 0 && (((uintptr_t)in | (uintptr_t)out) & 15) == 0) {  // 16 bytes per access
    const int per = d / VEC;
    for (int i = threadIdx.x; i < H * per; i += blockDim.x) {
      const int h = i / per, c = i - h * per;
      uint4 raw = *reinterpret_cast<const uint4*>(in + ((size_t)h * N + b) * d + c * VEC);
      if (gate.p) {
        const float s = row_sum_splits(gate.p + (size_t)n * gate.ld + h, gate.splits, gate.split_stride);
        const float den = 1.f + expf(-s);
        T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
        for (int u = 0; u < VEC; ++u) e[u] = from_f32<T>(to_f32<T>(e[u]) / den);
      }
      *reinterpret_cast<uint4*>(out + (size_t)n * H * d + (size_t)i * VEC) = raw;
    }
    return;
  }
  for (int i = threadIdx.x; i < H * d; i += blockDim.x) {
    const int h = i / d, c = i - h * d;
    T v = in[((size_t)h * N + b) * d + c];
    if (gate.p) {
      const float s = row_sum_splits(gate.p + (size_t)n * gate.ld + h, gate.splits, gate.split_stride);
      v = from_f32<T>(to_f32<T>(v) / (1.f + expf(-s)));
    }
    out[(size_t)n * H * d + i] = v;
  }
}

JLX_API int jlx_heads_to_rows(const void* in, void* out, int dtype, int N, int H, int d, const GateRowsView* gate, const int* rows,
                              cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && H > 0 && d > 0, "heads_to_rows: bad sizes");
  if (N == 0) return 0;
  const GateRowsView none = {nullptr, 0, 0, 1, 0};
  JLX_DISPATCH_DTYPE(dtype, T, {
    JLX_CUDA(jlx_launch_pdl(heads_to_rows_kernel<T>, dim3(N), dim3(256), 0, stream, (const T*)in, (T*)out, N, H, d, gate ? *gate : none, rows));
  });
  JLX_LAUNCH_CHECK("heads_to_rows");
  return 0;
}
