// Position encoding of q and k, weightless L2 norm of q and k, and the write of k and v into
// the paged cache, in one pass over a step's projected rows.
//
// Rotation: adjacent pairs (2j, 2j+1) turn by angle position * inv_freq[j]
// (llama4/llama4_jax/model.py:712-728); the angle, sine and cosine are 32-bit.  The norm follows the
// rotation (model.py:915-917) and divides by sqrt(mean(v^2) + eps) (model.py:885-888 with gamma None).
// Layers without position encoding pass inv_freq = null and l2norm = 0: their rows are copied.
//
// Cache layout of one layer: pages[page][0 = K, 1 = V][kv head][slot in page][dh].
#include "common.cuh"

#define ROPE_REG_PAIRS 4  // head sizes up to 256 keep a lane's pairs in registers

// A rotary pair (2j, 2j+1) as one access.
template <typename T> __device__ __forceinline__ float2 load_pair(const T* p);
template <> __device__ __forceinline__ float2 load_pair<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 load_pair<bf16>(const bf16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
template <typename T> __device__ __forceinline__ void store_pair(T* p, float a, float b);
template <> __device__ __forceinline__ void store_pair<float>(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
template <> __device__ __forceinline__ void store_pair<bf16>(bf16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

// TI: element type of the projected rows (the activation type, or float32 split-K partials that are
// added first); T: element type of q_out and of the cache.
// HPW: heads per warp.  A block takes 8 * HPW heads of one token (head h0 + 8 i for warp h0's i-th turn).  With many
// tokens a block's fixed chain of dependent loads (position, request, block table) is paid once for more heads,
// and a warp's loads of all its heads are in flight together; with few tokens one head per warp gives the most blocks.
template <typename TI, typename T, int HPW>
__global__ void __launch_bounds__(256)
rope_kv_store_kernel(const TI* __restrict__ qkv, int splits, long long split_stride, T* __restrict__ q_out,
                     T* __restrict__ pages, const int* __restrict__ block_table, int bt_stride,
                     const int* __restrict__ req_of_token, const int* __restrict__ positions,
                     const float* __restrict__ inv_freq, int l2norm, float eps, int Hq, int Hkv, int dh, int page_size,
                     int num_pages, int store_kv, int* status) {
  JLX_TL(TL_ROPE);
  extern __shared__ float sc[];  // [dh / 2][2]: sine and cosine of this token's angles
  pdl_launch_dependents();
  const int n = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int heads = Hq + 2 * Hkv;
  const int half = dh >> 1;
  const TI* row = qkv + (size_t)n * heads * dh;
  // What does not depend on the kernels before this one in the stream comes first: the token's position, its request
  // and page (the step's description, copied to the device before the step began), and the sines and cosines of
  // its angles.  The block starts while its predecessor still runs, so this chain of dependent loads and the
  // transcendental functions cost the step nothing; only the projected rows wait for the predecessor.
  const int pos = positions[n];
  T* kdst = nullptr;
  T* vdst = nullptr;
  if (store_kv) {
    const int r = req_of_token[n];
    const int page = block_table[(size_t)r * bt_stride + pos / page_size];
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, JLX_STATUS_BAD_PAGE);
    } else {
      T* base = pages + (size_t)page * 2 * Hkv * page_size * dh;
      kdst = base + (size_t)(pos % page_size) * dh;
      vdst = base + (size_t)Hkv * page_size * dh + (size_t)(pos % page_size) * dh;
    }
  }
  if (inv_freq) {
    for (int j = threadIdx.x; j < half; j += blockDim.x) sincosf((float)pos * inv_freq[j], &sc[2 * j], &sc[2 * j + 1]);
    __syncthreads();
  }
  // With the pairs kept in registers a warp's loads of all its heads are issued together.
  const int h0 = blockIdx.y * 8 * HPW + warp;
  const bool in_regs = half <= 32 * ROPE_REG_PAIRS;
  float va[HPW][ROPE_REG_PAIRS], vb[HPW][ROPE_REG_PAIRS];
  // A decode step's few blocks rehearse (see jlx_rehearses): the rest of the kernel runs once without its loads
  // and stores while the predecessor still works, and then for real.
#pragma unroll 1
  for (int pass = in_regs && jlx_rehearses() ? 0 : 1; pass < 2; ++pass) {
  const bool real = pass == 1;
  if (real) pdl_wait();
  if (in_regs) {
#pragma unroll
    for (int t = 0; t < HPW; ++t) {
      const int h = h0 + 8 * t;
      const TI* src = row + (size_t)h * dh;
#pragma unroll
      for (int i = 0; i < ROPE_REG_PAIRS; ++i) {
        const int j = lane + 32 * i;
        float a = 0.f, b = 0.f;
        if (real && h < heads && j < half) {
          // the split-K partials of a pair are fetched eight at a time and then added in ascending order: a loop
          // that added each as it came paid one memory latency per partial
          for (int z0 = 0; z0 < splits; z0 += 8) {
            float2 v[8];
#pragma unroll
            for (int u = 0; u < 8; ++u)
              if (z0 + u < splits) v[u] = load_pair<TI>(src + (size_t)(z0 + u) * split_stride + 2 * j);
#pragma unroll
            for (int u = 0; u < 8; ++u)
              if (z0 + u < splits) {
                if (z0 + u == 0) { a = v[u].x; b = v[u].y; }
                else { a += v[u].x; b += v[u].y; }
              }
          }
        }
        va[t][i] = a;
        vb[t][i] = b;
      }
    }
  }

  JLX_TL_MARK(0);
#pragma unroll
  for (int t = 0; t < HPW; ++t) {
    const int h = h0 + 8 * t;
    if (h >= heads) break;
    const TI* src = row + (size_t)h * dh;
    const bool is_v = h >= Hq + Hkv;  // value heads are copied (the sum of the partials): no rotation, no norm
    T* dst = h < Hq ? q_out + ((size_t)n * Hq + h) * dh
                    : (is_v ? (vdst ? vdst + (size_t)(h - Hq - Hkv) * page_size * dh : nullptr)
                            : (kdst ? kdst + (size_t)(h - Hq) * page_size * dh : nullptr));
    if (in_regs) {
      // one pass: a lane keeps its pairs in registers between the sum of squares and the write
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < ROPE_REG_PAIRS; ++i) {
        const int j = lane + 32 * i;
        if (j < half) {
          float a = va[t][i], b = vb[t][i];
          if (inv_freq && !is_v) {
            const float s = sc[2 * j], c = sc[2 * j + 1];
            const float ra = a * c - b * s, rb = b * c + a * s;
            a = ra;
            b = rb;
          }
          ss += a * a + b * b;
          va[t][i] = a;
          vb[t][i] = b;
        }
      }
      float inv = 1.f;
      if (l2norm && !is_v) {
        ss = warp_sum(ss);
        inv = 1.f / sqrtf(ss / (float)dh + eps);
      }
      if (!dst) continue;
#pragma unroll
      for (int i = 0; i < ROPE_REG_PAIRS; ++i) {
        const int j = lane + 32 * i;
        if (real && j < half) store_pair<T>(dst + 2 * j, va[t][i] * inv, vb[t][i] * inv);
      }
      continue;
    }
    if (is_v) {
      if (dst) {
        for (int j = lane; j < half; j += 32) {
          float a = 0.f, b = 0.f;
          for (int z = 0; z < splits; ++z) {
            const float2 v = load_pair<TI>(src + (size_t)z * split_stride + 2 * j);
            a += v.x;
            b += v.y;
          }
          store_pair<T>(dst + 2 * j, a, b);
        }
      }
      continue;
    }
    // larger heads: pass 1 rotates and accumulates the sum of squares
    float ss = 0.f;
    for (int j = lane; j < half; j += 32) {
      float a = 0.f, b = 0.f;
      for (int z = 0; z < splits; ++z) {
        a += to_f32<TI>(src[(size_t)z * split_stride + 2 * j]);
        b += to_f32<TI>(src[(size_t)z * split_stride + 2 * j + 1]);
      }
      if (inv_freq) {
        const float s = sc[2 * j], c = sc[2 * j + 1];
        const float ra = a * c - b * s, rb = b * c + a * s;
        a = ra;
        b = rb;
      }
      ss += a * a + b * b;
    }
    float inv = 1.f;
    if (l2norm) {
      ss = warp_sum(ss);
      inv = 1.f / sqrtf(ss / (float)dh + eps);
    }
    if (!dst) continue;
    // pass 2: the same values again, scaled and written
    for (int j = lane; j < half; j += 32) {
      float a = 0.f, b = 0.f;
      for (int z = 0; z < splits; ++z) {
        a += to_f32<TI>(src[(size_t)z * split_stride + 2 * j]);
        b += to_f32<TI>(src[(size_t)z * split_stride + 2 * j + 1]);
      }
      if (inv_freq) {
        const float s = sc[2 * j], c = sc[2 * j + 1];
        const float ra = a * c - b * s, rb = b * c + a * s;
        a = ra;
        b = rb;
      }
      dst[2 * j] = from_f32<T>(a * inv);
      dst[2 * j + 1] = from_f32<T>(b * inv);
    }
  }
  }
}

// The same for many tokens in bfloat16 (a prompt portion): one block per token takes ALL its heads, eight elements
// (four rotary pairs, 16 bytes) per thread and access, so that a token's angles are computed once (not once per
// group of heads) and every load and store is 16 bytes wide.  A head's dh / 8 threads are neighbours in a warp and
// add their squares by shuffles.  Needs dh / 8 a power of two up to 32 (head sizes 8, 16, 32, 64, 128, 256).
// The arithmetic of an element is the general kernel's; only the order of the sum of squares differs.
__global__ void __launch_bounds__(256)
rope_kv_store_rows_kernel(const bf16* __restrict__ qkv, bf16* __restrict__ q_out, bf16* __restrict__ pages,
                          const int* __restrict__ block_table, int bt_stride, const int* __restrict__ req_of_token,
                          const int* __restrict__ positions, const float* __restrict__ inv_freq, int l2norm, float eps, int Hq,
                          int Hkv, int dh, int page_size, int num_pages, int store_kv, int* status) {
  JLX_TL(TL_ROPE);
  extern __shared__ float sc[];  // [dh / 2][2]: sine and cosine of this token's angles
  pdl_launch_dependents();
  pdl_wait();
  const int n = blockIdx.x;
  const int heads = Hq + 2 * Hkv, per_head = dh >> 3, vectors = heads * per_head;
  const uint4* row = reinterpret_cast<const uint4*>(qkv + (size_t)n * heads * dh);
  // this thread's vectors first: the loads depend on nothing and fly during the dependent loads below
  constexpr int MAXV = 4;
  uint4 v[MAXV];
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int idx = threadIdx.x + i * 256;
    if (idx < vectors) v[i] = row[idx];
  }
  const int pos = positions[n];
  bf16* kdst = nullptr;
  bf16* vdst = nullptr;
  if (store_kv) {
    const int r = req_of_token[n];
    const int page = block_table[(size_t)r * bt_stride + pos / page_size];
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, JLX_STATUS_BAD_PAGE);
    } else {
      bf16* base = pages + (size_t)page * 2 * Hkv * page_size * dh;
      kdst = base + (size_t)(pos % page_size) * dh;
      vdst = base + (size_t)Hkv * page_size * dh + (size_t)(pos % page_size) * dh;
    }
  }
  if (inv_freq) {
    for (int j = threadIdx.x; j < (dh >> 1); j += blockDim.x) sincosf((float)pos * inv_freq[j], &sc[2 * j], &sc[2 * j + 1]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int idx = threadIdx.x + i * 256;
    const bool mine = idx < vectors;  // (no early exit: the shuffles below need the whole warp)
    const int h = mine ? idx / per_head : 0, part = idx % per_head;
    const bool is_v = h >= Hq + Hkv;
    float f[8];
    {
      const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&v[i]);
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float2 t = mine ? __bfloat1622float2(p2[u]) : make_float2(0.f, 0.f);
        f[2 * u] = t.x;
        f[2 * u + 1] = t.y;
      }
    }
    float ss = 0.f;
    if (!is_v) {
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        float a = f[2 * u], b = f[2 * u + 1];
        if (inv_freq) {
          const int j = part * 4 + u;
          const float s = sc[2 * j], c = sc[2 * j + 1];
          const float ra = a * c - b * s, rb = b * c + a * s;
          a = ra;
          b = rb;
        }
        ss += a * a + b * b;
        f[2 * u] = a;
        f[2 * u + 1] = b;
      }
    }
    float inv = 1.f;
    if (l2norm) {  // uniform over the block
      for (int o = per_head >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (!is_v) inv = 1.f / sqrtf(ss / (float)dh + eps);
    }
    if (!mine) continue;
    bf16* dst = h < Hq ? q_out + ((size_t)n * Hq + h) * dh
                       : (is_v ? (vdst ? vdst + (size_t)(h - Hq - Hkv) * page_size * dh : nullptr)
                               : (kdst ? kdst + (size_t)(h - Hq) * page_size * dh : nullptr));
    if (!dst) continue;
    uint4 o;
    if (is_v) {
      o = v[i];  // values are copied as they are
    } else {
      __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
      for (int u = 0; u < 4; ++u) o2[u] = __floats2bfloat162_rn(f[2 * u] * inv, f[2 * u + 1] * inv);
    }
    *reinterpret_cast<uint4*>(dst + part * 8) = o;
  }
}

JLX_API int jlx_rope_kv_store(const void* qkv, int in_dtype, int splits, long long split_stride, void* q_out, void* pages,
                              int dtype, const int* block_table, int bt_stride, const int* req_of_token,
                              const int* positions, const float* inv_freq, int l2norm, float eps, int N, int Hq, int Hkv,
                              int dh, int page_size, int num_pages, int store_kv, int* status, cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && Hq > 0 && Hkv >= 0 && dh > 0, "rope_kv_store: bad sizes N=%d Hq=%d Hkv=%d dh=%d", N, Hq, Hkv, dh);
  JLX_REQUIRE(dh % 2 == 0, "rope_kv_store: head size %d must be even (rotary pairs)", dh);
  JLX_REQUIRE(dh <= 8192, "rope_kv_store: head size %d is above the supported maximum 8192", dh);
  JLX_REQUIRE(!store_kv || (page_size > 0 && num_pages > 0 && bt_stride > 0), "rope_kv_store: bad cache sizes");
  JLX_REQUIRE(splits >= 1 && (splits == 1 || in_dtype == JLX_F32), "rope_kv_store: split-K partials are float32");
  JLX_REQUIRE((Hq + 2 * Hkv + 7) / 8 <= 65535, "rope_kv_store: too many heads");
  if (N == 0) return 0;
  const size_t smem = (size_t)dh * sizeof(float);
  const int heads = Hq + 2 * Hkv;
  // many tokens (prompt portions): two heads per warp; few (decoding): one, for the most blocks
  const bool wide = N >= 256 && heads > 8;
  // many tokens in bfloat16: the kernel that takes a token's heads 16 bytes at a time
  const int per_head = dh / 8;
  if (N >= 256 && in_dtype == JLX_BF16 && dtype == JLX_BF16 && splits == 1 && dh % 8 == 0 && per_head <= 32 &&
      (per_head & (per_head - 1)) == 0 && heads * per_head <= 4 * 256 &&
      (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)pages) & 15) == 0) {
    JLX_CUDA(jlx_launch_pdl(rope_kv_store_rows_kernel, dim3(N), dim3(256), smem, stream, (const bf16*)qkv, (bf16*)q_out,
                            (bf16*)pages, block_table, bt_stride, req_of_token, positions, inv_freq, l2norm, eps, Hq, Hkv, dh,
                            page_size, num_pages, store_kv, status));
    return 0;
  }
  JLX_DISPATCH_DTYPE(in_dtype, TI, JLX_DISPATCH_DTYPE(dtype, T, {
    if (wide) {
      JLX_CUDA(jlx_launch_pdl(rope_kv_store_kernel<TI, T, 2>, dim3(N, (heads + 15) / 16), dim3(256), smem, stream,
                              (const TI*)qkv, splits, split_stride, (T*)q_out, (T*)pages, block_table, bt_stride, req_of_token,
                              positions, inv_freq, l2norm, eps, Hq, Hkv, dh, page_size, num_pages, store_kv, status));
    } else {
      JLX_CUDA(jlx_launch_pdl(rope_kv_store_kernel<TI, T, 1>, dim3(N, (heads + 7) / 8), dim3(256), smem, stream,
                              (const TI*)qkv, splits, split_stride, (T*)q_out, (T*)pages, block_table, bt_stride, req_of_token,
                              positions, inv_freq, l2norm, eps, Hq, Hkv, dh, page_size, num_pages, store_kv, status));
    }
  }));
  return 0;
}

// Plain write of already-encoded k and v rows into pages (for position encodings that are not fused).
// k, v: [N, Hkv, dh]
template <typename T>
__global__ void kv_store_kernel(const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ pages,
                                const int* __restrict__ block_table, int bt_stride,
                                const int* __restrict__ req_of_token, const int* __restrict__ positions, int Hkv,
                                int dh, int page_size, int num_pages, int* status) {
  JLX_TL(TL_KV_STORE);
  const int n = blockIdx.x;
  const int pos = positions[n];
  const int page = block_table[(size_t)req_of_token[n] * bt_stride + pos / page_size];
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicOr(status, JLX_STATUS_BAD_PAGE);
    return;
  }
  T* base = pages + (size_t)page * 2 * Hkv * page_size * dh;
  for (int i = threadIdx.x; i < Hkv * dh; i += blockDim.x) {
    const int h = i / dh, d = i % dh;
    const size_t o = ((size_t)h * page_size + pos % page_size) * dh + d;
    base[o] = k[(size_t)n * Hkv * dh + i];
    base[(size_t)Hkv * page_size * dh + o] = v[(size_t)n * Hkv * dh + i];
  }
}

JLX_API int jlx_kv_store(const void* k, const void* v, void* pages, int dtype, const int* block_table, int bt_stride,
                         const int* req_of_token, const int* positions, int N, int Hkv, int dh, int page_size,
                         int num_pages, int* status, cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && Hkv > 0 && dh > 0 && page_size > 0 && num_pages > 0, "kv_store: bad sizes");
  if (N == 0) return 0;
  JLX_DISPATCH_DTYPE(dtype, T,
                     (kv_store_kernel<T><<<N, 128, 0, stream>>>((const T*)k, (const T*)v, (T*)pages, block_table,
                                                                bt_stride, req_of_token, positions, Hkv, dh, page_size,
                                                                num_pages, status)));
  JLX_LAUNCH_CHECK("kv_store");
  return 0;
}

// ------------------------------------------------------------------------------------------------------------------
// The same pass in a general form, for attention whose q and k are RMS-normed (with a weight or without) BEFORE or AFTER
// the rotation, rotated on their first rot_dims entries only, in halves or in neighbouring pairs, and whose values may
// have another size than its keys, or be the keys as projected.
//
//   norm:   y = x / sqrt(mean(x^2) + eps) (* w)   over the head's dk entries (w: [dk], shared by the heads, or null)
//   halves: (y_i, y_(i + rot/2)) <- (y_i cos a - y_(i + rot/2) sin a,  y_(i + rot/2) cos a + y_i sin a),
//   pairs:  (y_2i, y_(2i + 1))   <- (y_2i cos a - y_(2i + 1) sin a,    y_(2i + 1) cos a + y_2i sin a),
//           a = position * inv_freq[i], i < rot / 2; entries from rot on pass unchanged.  cos a and sin a are both
//           multiplied by `amplitude` (1: a plain rotation).
//
// The projected rows are float32 (split-K partials are added first) with the q heads from column 0, the k heads from
// column k_col and the v heads (dv entries each) from column v_col (v_col = k_col: the values are the keys as they
// were projected).  q_out and the cache keep `dpad` entries per head: keys, queries and values are padded with zeros
// up to it, so that one page layout and the attention kernels built for equal sizes serve keys of one size and values
// of another.
//
// `bias` (float32, one number per projected column, or null) is added to the projected rows first.  With `maps` = 2 the q and
// k heads are pairs of maps over the values of one head: Hq and Hkv count q rows and VALUE heads, the 2 Hkv keys of dk
// entries lie head by head as [map 1, map 2] and go side by side into one cached row, and a query row holds its map's
// entries at that map's place, zeros elsewhere (see attention_maps.cuh).
enum { ROPE_PAIRS_HALVES = 0, ROPE_PAIRS_INTERLEAVED = 1 };
// ROPE_NORM_WHOLE: before the rotation, over ALL heads of the projection at once: q / sqrt(mean over its Hq dk entries
// + eps) * w, w: [Hq dk] ([Hkv dk] for k).
enum { ROPE_NORM_NONE = 0, ROPE_NORM_BEFORE = 1, ROPE_NORM_AFTER = 2, ROPE_NORM_WHOLE = 3 };

struct RopeRowsView {
  const float* p;
  long long split_stride;
  long long ld;
  int splits;
  int pad_;
};

template <typename T>
__global__ void rope_half_kv_store_kernel(RopeRowsView proj, int k_col, int v_col, T* __restrict__ q_out, T* __restrict__ pages,
                                          const int* __restrict__ block_table, int bt_stride, const int* __restrict__ req_of_token,
                                          const int* __restrict__ positions, const float* __restrict__ q_norm_w,
                                          const float* __restrict__ k_norm_w, float eps, const float* __restrict__ inv_freq,
                                          int rot, int pairing, int norm_mode, int Hq, int Hkv, int dk, int dv, int dpad,
                                          int page_size, int num_pages, int store, int* status, float amplitude, const float* __restrict__ q_scale,
                                          int v_norm, const float* __restrict__ bias, int maps) {
  JLX_TL(TL_ROPE);
  pdl_launch_dependents_if_small();
  __shared__ float whole_part[2][8];
  extern __shared__ float buf[];  // [warps][2][max(dk, dv)]: a head's row as projected (and normed), and as rotated; the angles
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
  const size_t n = blockIdx.x;
  const int dmax = dk > dv ? dk : dv;
  float* row = buf + (size_t)warp * 2 * dmax;
  float* turned = row + dmax;
  float* angles = buf + (size_t)nwarp * 2 * dmax;  // [rot / 2][2]: sine and cosine of this token's angles
  // the step's description is older than the step: the token's place and its angles are made before the wait for the
  // projected rows
  const int pos = positions[n];
  const int half = rot >> 1;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * inv_freq[i], &sn, &cs);
    angles[2 * i] = sn * amplitude;
    angles[2 * i + 1] = cs * amplitude;
  }
  T* kdst = nullptr;
  if (store) {
    const int page = block_table[(size_t)req_of_token[n] * bt_stride + pos / page_size];
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, JLX_STATUS_BAD_PAGE);
    } else {
      kdst = pages + ((size_t)page * 2 * Hkv * page_size + (size_t)(pos % page_size)) * dpad;
    }
  }
  __syncthreads();
  pdl_wait();
  const int n_k = maps * Hkv;  // keys that the token projects
  const int heads = Hq + (store ? n_k + Hkv : 0);
  float whole_rms[2] = {1.f, 1.f};  // of all q entries, of all k entries
  if (norm_mode == ROPE_NORM_WHOLE) {
    // every block of the token makes both sums itself, in an order fixed by the block's size (the model's head count)
    for (int which = 0; which < (store ? 2 : 1); ++which) {
      const int cnt = (which ? n_k : Hq) * dk, col0 = which ? k_col : 0;
      float ss = 0.f;
      for (int i = threadIdx.x; i < cnt; i += blockDim.x) {
        float v = 0.f;
        for (int z = 0; z < proj.splits; ++z) v += proj.p[(size_t)z * proj.split_stride + n * proj.ld + col0 + i];
        if (bias) v += bias[col0 + i];
        ss = fmaf(v, v, ss);
      }
      ss = warp_sum(ss);
      if (lane == 0) whole_part[which][warp] = ss;
    }
    __syncthreads();
    for (int which = 0; which < (store ? 2 : 1); ++which) {
      float ss = 0.f;
      for (int w = 0; w < nwarp; ++w) ss += whole_part[which][w];
      whole_rms[which] = sqrtf(ss / (float)((which ? n_k : Hq) * dk) + eps);
    }
  }
  for (int hh = blockIdx.y * nwarp + warp; hh < heads; hh += gridDim.y * nwarp) {
    const bool is_q = hh < Hq, is_k = !is_q && hh < Hq + n_k;
    const bool qk = is_q || is_k;
    const int d = qk ? dk : dv;
    const int col = is_q ? hh * dk : (is_k ? k_col + (hh - Hq) * dk : v_col + (hh - Hq - n_k) * dv);
    // where the head's entries go in its row of dpad, and which stretch of the row this warp writes
    int at = 0, w_lo = 0, w_hi = dpad;
    T* dst;
    if (is_q) {
      dst = q_out + (n * Hq + hh) * dpad;
      at = (hh % maps) * dk;
    } else if (!kdst) {
      continue;
    } else if (is_k) {
      const int map = (hh - Hq) % maps;
      dst = kdst + (size_t)((hh - Hq) / maps) * page_size * dpad;
      at = w_lo = map * dk;
      if (map + 1 < maps) w_hi = w_lo + dk;  // the last map's warp writes the padding
    } else {
      dst = kdst + (size_t)(Hkv + hh - Hq - n_k) * page_size * dpad;
    }
    float ss = 0.f;
    for (int i = lane; i < d; i += 32) {
      float s = 0.f;
      for (int z = 0; z < proj.splits; ++z) s += proj.p[(size_t)z * proj.split_stride + n * proj.ld + col + i];
      if (bias) s += bias[col + i];
      row[i] = s;
      ss = fmaf(s, s, ss);
    }
    const float* w = is_q ? q_norm_w : (is_k ? k_norm_w : nullptr);
    if ((qk && norm_mode == ROPE_NORM_BEFORE) || (!qk && v_norm)) {
      ss = warp_sum(ss);
      const float rms = sqrtf(ss / (float)d + eps);
      __syncwarp();
      for (int i = lane; i < d; i += 32) row[i] = w ? row[i] / rms * w[i] : row[i] / rms;
    } else if (qk && norm_mode == ROPE_NORM_WHOLE) {
      const float rms = whole_rms[is_q ? 0 : 1];
      const float* wh = w ? w + (size_t)(is_q ? hh : hh - Hq) * dk : nullptr;  // the weight covers the whole projection
      __syncwarp();
      for (int i = lane; i < d; i += 32) row[i] = wh ? row[i] / rms * wh[i] : row[i] / rms;
    }
    __syncwarp();
    float ss2 = 0.f;
    for (int i = lane; i < d; i += 32) {
      float y = row[i];
      if (qk && i < rot) {
        // the entry's partner and which of the pair it is: (i, i + rot/2) side by side in halves, or (2j, 2j + 1)
        const bool first = pairing == ROPE_PAIRS_INTERLEAVED ? !(i & 1) : i < half;
        const int f = pairing == ROPE_PAIRS_INTERLEAVED ? i >> 1 : (first ? i : i - half);
        const int partner = pairing == ROPE_PAIRS_INTERLEAVED ? i ^ 1 : (first ? i + half : i - half);
        const float sn = angles[2 * f], cs = angles[2 * f + 1];
        y = first ? row[i] * cs - row[partner] * sn : row[i] * cs + row[partner] * sn;
      }
      turned[i] = y;
      ss2 = fmaf(y, y, ss2);
    }
    float rms_turned = 1.f;
    const bool after = qk && norm_mode == ROPE_NORM_AFTER;
    if (after) {
      ss2 = warp_sum(ss2);
      rms_turned = sqrtf(ss2 / (float)d + eps);
    }
    __syncwarp();
    const float qs = is_q && q_scale ? q_scale[hh] : 1.f;
    for (int j = w_lo + lane; j < w_hi; j += 32) {
      const int i = j - at;
      float y = 0.f;
      if (i >= 0 && i < d) {
        y = turned[i];
        if (after) y = w ? y / rms_turned * w[i] : y / rms_turned;
        y *= qs;
      }
      dst[j] = from_f32<T>(y);
    }
    __syncwarp();
  }
}

// The same for many tokens (a prompt portion) in bfloat16 without a norm, rotated in halves or not at all: one block per token,
// four neighbouring entries of a head's row per thread and access (16 bytes in, 8 out), so that a token's angles are made once
// and nothing passes through shared memory but them.  Needs sizes, columns and the half of the rotation in fours.
__global__ void __launch_bounds__(256)
rope_half_rows_kernel(RopeRowsView proj, int k_col, int v_col, bf16* __restrict__ q_out, bf16* __restrict__ pages, const int* __restrict__ block_table,
                      int bt_stride, const int* __restrict__ req_of_token, const int* __restrict__ positions, const float* __restrict__ inv_freq, int rot,
                      int Hq, int Hkv, int dk, int dv, int dpad, int page_size, int num_pages, int store, int* status, float amplitude,
                      const float* __restrict__ q_scale, const float* __restrict__ bias, int maps) {
  JLX_TL(TL_ROPE);
  pdl_launch_dependents_if_small();
  extern __shared__ __align__(16) float angles_s[];  // [2][rot / 2]: sines, then cosines, of this token's angles
  const size_t n = blockIdx.x;
  const int pos = positions[n], half = rot >> 1;
  float* sn = angles_s;
  float* cs = angles_s + half;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf((float)pos * inv_freq[i], &s, &c);
    sn[i] = s * amplitude;
    cs[i] = c * amplitude;
  }
  bf16* kdst = nullptr;
  if (store) {
    const int page = block_table[(size_t)req_of_token[n] * bt_stride + pos / page_size];
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, JLX_STATUS_BAD_PAGE);
    } else {
      kdst = pages + ((size_t)page * 2 * Hkv * page_size + (size_t)(pos % page_size)) * dpad;
    }
  }
  __syncthreads();
  pdl_wait();
  const float* row = proj.p + n * proj.ld;
  const int quads = dpad >> 2, rows = Hq + (kdst ? 2 * Hkv : 0);
  auto fetch = [&](int col) {  // four projected entries: partial sums added in order, then the bias
    float4 v = *reinterpret_cast<const float4*>(row + col);
    for (int z = 1; z < proj.splits; ++z) {
      const float4 w = *reinterpret_cast<const float4*>(row + (size_t)z * proj.split_stride + col);
      v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
    }
    if (bias) {
      const float4 b = *reinterpret_cast<const float4*>(bias + col);
      v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
    }
    return v;
  };
  for (int idx = threadIdx.x; idx < rows * quads; idx += blockDim.x) {
    const int r = idx / quads, j = (idx - r * quads) * 4;  // output row (a query row, a cached key row, a value row), first entry
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    bf16* dst;
    int col = -1, i = j;  // column of the entries, and their place in their map
    if (r < Hq) {
      dst = q_out + (n * Hq + r) * dpad;
      i = j - (r % maps) * dk;
      if (i >= 0 && i < dk) col = r * dk + i;
    } else if (r < Hq + Hkv) {
      dst = kdst + (size_t)(r - Hq) * page_size * dpad;
      if (j < maps * dk) {
        col = k_col + (r - Hq) * maps * dk + j;
        i = j % dk;
      }
    } else {
      dst = kdst + (size_t)(r - Hq) * page_size * dpad;
      if (j < dv) col = v_col + (r - Hq - Hkv) * dv + j;
      i = rot;  // values do not turn
    }
    if (col >= 0) {
      y = fetch(col);
      if (i < rot) {
        const bool first = i < half;
        const int f = first ? i : i - half;
        const float4 w = fetch(first ? col + half : col - half);
        const float4 s = *reinterpret_cast<const float4*>(sn + f), c = *reinterpret_cast<const float4*>(cs + f);
        const float g = first ? -1.f : 1.f;
        y = make_float4(y.x * c.x + g * w.x * s.x, y.y * c.y + g * w.y * s.y, y.z * c.z + g * w.z * s.z, y.w * c.w + g * w.w * s.w);
      }
      if (r < Hq && q_scale) {
        const float m = q_scale[r];
        y.x *= m; y.y *= m; y.z *= m; y.w *= m;
      }
    }
    uint2 o;
    *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(y.x, y.y);
    *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(y.z, y.w);
    *reinterpret_cast<uint2*>(dst + j) = o;
  }
}

// proj: float32 rows (see RopeRowsView; p points at the first q column).  pages: [P, 2, Hkv, page_size, dpad] or null.
// pairing: which entries turn together; norm_mode: no q/k norm, before the rotation, or after it (a null weight: the
// norm without one).  v_norm: each value head is divided by its root mean square over dv (no weight).  q_scale [Hq] (or
// null): every query head is multiplied by its number, last.  v_col == k_col with dv == dk stores the keys as projected (neither normed nor turned) as values.
JLX_API int jlx_rope_half_kv_store(const RopeRowsView* proj, int k_col, int v_col, void* q_out, void* pages, int dtype,
                                   const int* block_table, int bt_stride, const int* req_of_token, const int* positions,
                                   const float* q_norm_w, const float* k_norm_w, float eps, const float* inv_freq, int rot,
                                   int pairing, int norm_mode, int N, int Hq, int Hkv, int dk, int dv, int dpad, int page_size,
                                   int num_pages, int store, int* status, float amplitude, const float* q_scale, int v_norm,
                                   const float* bias, int maps, cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && Hq > 0 && Hkv > 0 && dk > 0 && dv > 0, "rope_half: bad sizes");
  JLX_REQUIRE(maps == 1 || (maps == 2 && Hq % 2 == 0 && norm_mode != ROPE_NORM_WHOLE && v_col != k_col), "rope_half: %d maps per head with %d query rows", maps, Hq);
  JLX_REQUIRE(dpad >= maps * dk && dpad >= dv, "rope_half: the padded head size %d is below the key or value size (%d, %d)", dpad, dk, dv);
  JLX_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= dk, "rope_half: %d rotated entries of %d", rot, dk);
  JLX_REQUIRE(rot == 0 || inv_freq, "rope_half: frequencies missing");
  JLX_REQUIRE(pairing == ROPE_PAIRS_HALVES || pairing == ROPE_PAIRS_INTERLEAVED, "rope_half: unknown pairing %d", pairing);
  JLX_REQUIRE(norm_mode >= ROPE_NORM_NONE && norm_mode <= ROPE_NORM_WHOLE, "rope_half: unknown norm mode %d", norm_mode);
  JLX_REQUIRE(!store || (pages && block_table && page_size > 0 && num_pages > 0), "rope_half: cache missing");
  if (N == 0) return 0;
  const bool in_fours = dk % 4 == 0 && dv % 4 == 0 && dpad % 4 == 0 && k_col % 4 == 0 && v_col % 4 == 0 && rot % 8 == 0 && proj->ld % 4 == 0 &&
                        proj->split_stride % 4 == 0 &&
                        (((uintptr_t)proj->p | (uintptr_t)q_out | (uintptr_t)pages | (uintptr_t)bias) & 15) == 0;
  if (N >= 64 && dtype == JLX_BF16 && norm_mode == ROPE_NORM_NONE && !v_norm && (pairing == ROPE_PAIRS_HALVES || rot == 0) && in_fours && rot <= 4096) {
    JLX_CUDA(jlx_launch_pdl(rope_half_rows_kernel, dim3(N), dim3(256), (size_t)rot * sizeof(float), stream, *proj, k_col, v_col, (bf16*)q_out, (bf16*)pages,
                            block_table, bt_stride, req_of_token, positions, inv_freq, rot, Hq, Hkv, dk, dv, dpad, page_size, num_pages, store, status,
                            amplitude, q_scale, bias, maps));
    JLX_LAUNCH_CHECK("rope_half_rows");
    return 0;
  }
  const int heads = Hq + (store ? (maps + 1) * Hkv : 0);
  const int nwarp = heads < 8 ? heads : 8;
  const int by = N >= 64 ? 1 : (heads + nwarp - 1) / nwarp;
  const size_t smem = sizeof(float) * (2 * (size_t)nwarp * (dk > dv ? dk : dv) + rot);
  JLX_REQUIRE(smem <= 48 * 1024, "rope_half: head size too large");
  JLX_DISPATCH_DTYPE(dtype, T, {
    JLX_CUDA(jlx_launch_pdl(rope_half_kv_store_kernel<T>, dim3(N, by), dim3(nwarp * 32), smem, stream, *proj, k_col, v_col,
                            (T*)q_out, (T*)pages, block_table, bt_stride, req_of_token, positions, q_norm_w, k_norm_w, eps,
                            inv_freq, rot, pairing, norm_mode, Hq, Hkv, dk, dv, dpad, page_size, num_pages, store, status, amplitude,
                            q_scale, v_norm, bias, maps));
  });
  JLX_LAUNCH_CHECK("rope_half_kv_store");
  return 0;
}

// out[n, h dv + c] = mult * sigmoid(gate[n, h]) * attn[n, h, c], c < dv: the attention's heads (dpad entries each, of
// which dv count) through a gate per token and head, into (a column range of) the rows that the output product reads.
// gate: float32 rows, possibly split-K partials (p null: no gate).
template <typename T>
__global__ void head_gate_kernel(const T* __restrict__ attn, RopeRowsView gate, int per_channel, float mult, T* __restrict__ out,
                                 long long ld_out, int Hq, int dv, int dpad) {
  JLX_TL(TL_OTHER);
  pdl_launch_dependents_if_small();
  pdl_wait();
  const size_t n = blockIdx.x;
  for (int idx = threadIdx.x; idx < Hq * dv; idx += blockDim.x) {
    const int hd = idx / dv, c = idx - hd * dv;
    float g = mult;
    if (gate.p) {
      float s = 0.f;
      for (int z = 0; z < gate.splits; ++z) s += gate.p[(size_t)z * gate.split_stride + n * gate.ld + (per_channel ? idx : hd)];
      g *= 1.f / (1.f + expf(-s));
    }
    out[n * ld_out + idx] = from_f32<T>(g * to_f32<T>(attn[(n * Hq + hd) * dpad + c]));
  }
}

JLX_API int jlx_head_gate(const void* attn, const RopeRowsView* gate, int per_channel, float mult, void* out, int dtype,
                          long long ld_out, int N, int Hq, int dv, int dpad, cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && Hq > 0 && dv > 0 && dpad >= dv && ld_out >= (long long)Hq * dv, "head_gate: bad sizes");
  if (N == 0) return 0;
  RopeRowsView none = {nullptr, 0, 0, 1, 0};
  JLX_DISPATCH_DTYPE(dtype, T, {
    JLX_CUDA(jlx_launch_pdl(head_gate_kernel<T>, dim3(N), dim3(Hq * dv >= 1024 ? 256 : 128), 0, stream, (const T*)attn,
                            gate ? *gate : none, per_channel, mult, (T*)out, ld_out, Hq, dv, dpad));
  });
  JLX_LAUNCH_CHECK("head_gate");
  return 0;
}
