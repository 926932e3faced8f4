// Paged attention for any head size, head count, group size, page size and query length, in 32-bit
// or bfloat16 storage with 32-bit scores, softmax and accumulation.  It is the attention of the
// 32-bit path and the fallback of the bfloat16 path for sizes that the tensor-core kernels refuse.
//
// One block serves one query token and one KV head (all G query heads of the group share each key
// and value tile).  A query at position p of request r attends keys at positions [start, p] with
//   start = max(chunk  ? floor(p / chunk) * chunk : 0,  window ? p - window + 1 : 0)
// (causal and same-chunk mask of llama4/llama4_jax/model.py:731-742; scale dh^-0.5, model.py:774;
// 32-bit softmax, model.py:789).  Queries of layers with temperature tuning are scaled by
// 1 + attn_scale * ln(1 + floor((p + 1) / floor_scale)).
// With `keep` > 0 (and a window) the first `keep` keys of the sequence are visible besides the window's.
// With `sink` (one number per query head) the softmax has one more term in its denominator, exp(sink[h]), which
// carries no value: weights p_j = exp(s_j) / (exp(sink) + sum_i exp(s_i)); a sink of 0 adds one to the denominator.
// With `slopes` (one number per query head) slopes[h] * (p - j) is taken off the scaled score of key j: a bias that
// grows with the distance.
// With `softcap` > 0 the scaled score s becomes softcap * tanh(s / softcap) (before the bias and the sink).
// The order of the key loop depends only on (start, p): a position's result does not change with
// what else is in the batch or how the prompt was cut into steps.
#include "attention_maps.cuh"
#include "common.cuh"

#define ATT_TILE 32
#define ATT_MAX_WARPS 8
#define ATT_MAX_D32 16  // head size up to 512

template <typename T, typename TO>
__global__ void attention_generic_kernel(const T* __restrict__ q, const T* __restrict__ pages,
                                         const int* __restrict__ block_table, int bt_stride,
                                         const int* __restrict__ req_of_token, const int* __restrict__ positions,
                                         TO* __restrict__ out, int Hq, int Hkv, int dh, int page_size, int num_pages,
                                         float scale, int chunk, int window, int keep, float attn_scale, float floor_scale,
                                         const float* __restrict__ sink, const float* __restrict__ slopes, float softcap,
                                         int* status) {
  JLX_TL(TL_ATTN_GENERIC);
  extern __shared__ float smem[];
  const int n = blockIdx.x, hk = blockIdx.y;
  const int G = Hq / Hkv;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
  const int ldk = dh + 1;
  float* qs = smem;                        // [nwarp][dh]
  float* ks = qs + nwarp * dh;             // [ATT_TILE][dh + 1]
  float* vs = ks + ATT_TILE * ldk;         // [ATT_TILE][dh + 1]

  const int p = positions[n];
  const int r = req_of_token[n];
  int start = 0;
  if (chunk > 0) start = (p / chunk) * chunk;
  if (window > 0) start = max(start, p - window + 1);
  const int kept = min(keep, start);  // kept keys below the window
  float qscale = scale;
  if (attn_scale != 0.f) qscale *= 1.f + attn_scale * log1pf(floorf(((float)p + 1.f) / floor_scale));
  const int nd = (dh + 31) >> 5;
  const size_t page_elems = (size_t)2 * Hkv * page_size * dh;

  for (int g0 = 0; g0 < G; g0 += nwarp) {
    const int g = g0 + warp;
    const bool active = g < G;
    const int h = hk * G + g;
    if (active)
      for (int d = lane; d < dh; d += 32) qs[warp * dh + d] = to_f32<T>(q[((size_t)n * Hq + h) * dh + d]);
    const float slope = slopes && active ? slopes[h] : 0.f;
    float m = -INFINITY, l = 0.f;
    float acc[ATT_MAX_D32];
#pragma unroll
    for (int i = 0; i < ATT_MAX_D32; ++i) acc[i] = 0.f;

    int t0 = kept > 0 ? 0 : start;
    while (t0 <= p) {
      __syncthreads();  // previous tile fully consumed; qs visible
      const int cnt = min(ATT_TILE, t0 < start ? kept - t0 : p - t0 + 1);
      for (int idx = threadIdx.x; idx < cnt * dh; idx += blockDim.x) {
        const int j = idx / dh, d = idx - j * dh;
        const int pos = t0 + j;
        const int page = block_table[(size_t)r * bt_stride + pos / page_size];
        float kv = 0.f, vv = 0.f;
        if (page < 0 || page >= num_pages) {
          atomicOr(status, JLX_STATUS_BAD_PAGE);
        } else {
          const T* base = pages + (size_t)page * page_elems + ((size_t)hk * page_size + pos % page_size) * dh + d;
          kv = to_f32<T>(base[0]);
          vv = to_f32<T>(base[(size_t)Hkv * page_size * dh]);
        }
        ks[j * ldk + d] = kv;
        vs[j * ldk + d] = vv;
      }
      __syncthreads();
      if (active) {
        float s = -INFINITY;
        if (lane < cnt) {
          float dot = 0.f;
          const float* kr = ks + lane * ldk;
          const float* qr = qs + warp * dh;
          for (int d = 0; d < dh; ++d) dot += qr[d] * kr[d];
          s = dot * qscale;
          if (softcap > 0.f) s = softcap * tanhf(s / softcap);
          s = fmaf(-slope, (float)(p - (t0 + lane)), s);
        }
        const float m_new = fmaxf(m, warp_max(s));
        const float corr = expf(m - m_new);  // m = -inf on the first tile: exp(-inf) = 0
        const float pj = lane < cnt ? expf(s - m_new) : 0.f;
        l = l * corr + warp_sum(pj);
        m = m_new;
#pragma unroll
        for (int i = 0; i < ATT_MAX_D32; ++i) {
          if (i < nd) {
            const int d = lane + 32 * i;
            float a = acc[i] * corr;
            for (int j = 0; j < cnt; ++j) {
              const float pv = __shfl_sync(0xffffffffu, pj, j);
              if (d < dh) a += pv * vs[j * ldk + d];
            }
            acc[i] = a;
          }
        }
      }
      t0 += ATT_TILE;
      if (t0 - ATT_TILE < start && t0 >= kept) t0 = start;  // the kept keys are through: on to the window
    }
    if (active) {
      float corr = 1.f;
      if (sink) {  // the sink joins the sum like a last key without a value
        const float m_new = fmaxf(m, sink[h]);
        corr = expf(m - m_new);
        l = l * corr + expf(sink[h] - m_new);
      }
#pragma unroll
      for (int i = 0; i < ATT_MAX_D32; ++i) {
        const int d = lane + 32 * i;
        if (i < nd && d < dh) out[((size_t)n * Hq + h) * dh + d] = from_f32<TO>(acc[i] * corr / l);
      }
    }
    __syncthreads();
  }
}

JLX_API int jlx_attention_generic(const void* q, const void* pages, int dtype, const int* block_table, int bt_stride,
                                  const int* req_of_token, const int* positions, void* out, int out_dtype, int N, int Hq, int Hkv,
                                  int dh, int page_size, int num_pages, float scale, int chunk, int window, int keep,
                                  float attn_scale, float floor_scale, const float* sink, const float* slopes,
                                  float softcap, int* status, cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && Hq > 0 && Hkv > 0 && dh > 0 && page_size > 0 && num_pages > 0, "attention: bad sizes");
  JLX_REQUIRE(Hq % Hkv == 0, "attention: %d query heads are no multiple of %d KV heads", Hq, Hkv);
  JLX_REQUIRE(dh <= 32 * ATT_MAX_D32, "attention: head size %d is above the supported maximum %d", dh, 32 * ATT_MAX_D32);
  JLX_REQUIRE(softcap >= 0.f, "attention: the score cap must be positive (0: none)");
  JLX_REQUIRE(attn_scale == 0.f || floor_scale > 0.f, "attention: floor_scale must be positive");
  if (N == 0) return 0;
  const int G = Hq / Hkv;
  const int nwarp = G < ATT_MAX_WARPS ? G : ATT_MAX_WARPS;
  const size_t smem = sizeof(float) * ((size_t)nwarp * dh + 2 * (size_t)ATT_TILE * (dh + 1));
  JLX_REQUIRE(Hkv <= 65535, "attention: too many KV heads (%d)", Hkv);
  JLX_REQUIRE(keep >= 0, "attention: the count of kept first keys is negative");
  JLX_DISPATCH_DTYPE(dtype, T, JLX_DISPATCH_DTYPE(out_dtype, TO, {
    if (smem > 48 * 1024)
      JLX_CUDA(cudaFuncSetAttribute(attention_generic_kernel<T, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attention_generic_kernel<T, TO><<<dim3(N, Hkv), nwarp * 32, smem, stream>>>(
        (const T*)q, (const T*)pages, block_table, bt_stride, req_of_token, positions, (TO*)out, Hq, Hkv, dh, page_size,
        num_pages, scale, chunk, window, keep, attn_scale, floor_scale, sink, slopes, softcap, status);
  }));
  JLX_LAUNCH_CHECK("attention_generic");
  return 0;
}

// The difference of two maps (see attention_maps.cuh) as a kernel of its own, behind the kernel above: attn float32
// [N, 2 H, dpad] -> out rows.  One warp per (token, head).
template <typename TO>
__global__ void map_difference_kernel(const float* __restrict__ attn, TO* __restrict__ out, MapDifference D, int items, int H, int dpad) {
  JLX_TL(TL_OTHER);
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= items) return;
  const int n = item / H, h = item - n * H;
  const float* a1 = attn + (size_t)item * 2 * dpad;
  const float* a2 = a1 + dpad;
  float ss = 0.f;
  for (int c = lane; c < D.out_dim; c += 32) {
    const float o = a1[c] - D.weight * a2[c];
    ss = fmaf(o, o, ss);
  }
  const float rms = sqrtf(warp_sum(ss) / (float)D.out_dim + D.eps);
  TO* dst = out + (size_t)n * D.ld_out + (size_t)h * D.out_dim;
  for (int c = lane; c < D.out_dim; c += 32) dst[c] = from_f32<TO>((a1[c] - D.weight * a2[c]) / rms * D.mult);
}

JLX_API int jlx_map_difference(const float* attn, void* out, int out_dtype, const MapDifference* diff, int N, int H, int dpad,
                               cudaStream_t stream) {
  JLX_REQUIRE(N >= 0 && H > 0 && diff && diff->out_dim > 0 && dpad >= diff->out_dim, "map_difference: bad sizes");
  if (N == 0) return 0;
  JLX_REQUIRE((long long)N * H < (1ll << 31), "map_difference: too many heads");
  const int items = N * H;
  JLX_DISPATCH_DTYPE(out_dtype, TO, {
    JLX_CUDA(jlx_launch_pdl(map_difference_kernel<TO>, dim3((items + 3) / 4), dim3(128), 0, stream, attn, (TO*)out, *diff, items, H, dpad));
  });
  JLX_LAUNCH_CHECK("map_difference");
  return 0;
}
