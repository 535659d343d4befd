// Decode attention (one new token per sequence, bfloat16) for mixers whose visible keys are the first
// `keep_first` positions of the sequence plus a window of the last positions (or all of them): the visible
// keys, counted in order (kept positions that lie before the window, then the window), are cut into chunks
// of 128; a block takes one chunk of one key/value head of one token and serves all query heads of that
// head, so that a key or value row is fetched once for the group; a second small launch merges the chunks.
//
// In a block each of eight warps takes 16 keys, two lanes a key: a lane reads half of its key's row in 16-byte pieces
// and makes that half of the dot products with every query head of the group (the queries lie in shared memory);
// one maximum and one correction per head for the warp's 16 keys; then the 16 value rows
// are walked through together, every lane owning a run of the value dims.  Both walks ask for several rows' pieces before
// they use the first, so that a block waits for memory a few times and not once a key.  Softmax, sums and accumulators are
// float32.  Partial results (m, l, acc[vd]) per (token, head, chunk) go to scratch that the caller gives.
// With `slopes` the score of key j loses slopes[head] * (p - j); with `sinks` the merge adds exp(sinks[head]) to the
// softmax's denominator (a term without a key or a value).  With `dist_bias` a score gains its head's entry for the
// distance to the key.
#include "common.cuh"

namespace {

constexpr int kWarps = 8;
constexpr int kWarpKeys = 16;
constexpr int kChunkKeys = kWarpKeys * kWarps;

// PER: query heads a key/value head (rounded up); DPL: value dims a lane (vd <= 32 * DPL, vd % DPL == 0)
template <int PER, int DPL>
__global__ void __launch_bounds__(32 * kWarps)
decode_kept_partial_kernel(const __nv_bfloat16* __restrict__ qkv, const __nv_bfloat16* __restrict__ kc,
                           const __nv_bfloat16* __restrict__ vc, float* __restrict__ part,
                           const int* __restrict__ positions, const int* __restrict__ seq_slot,
                           const int* __restrict__ pages, int max_blocks, int n_heads, int kv_heads, int hd, int vd,
                           float scale, int window, int keep_first, int n_chunks, const float* __restrict__ slopes, int chunk,
                           const float* __restrict__ head_scales, const float* __restrict__ dist_bias, int n_dist) {
  __shared__ __align__(16) float q_s[PER][256];
  __shared__ float m_s[kWarps][PER], l_s[kWarps][PER];
  __shared__ float acc_s[kWarps][PER][32 * DPL];
  const int c = blockIdx.x, g = blockIdx.y, t = blockIdx.z;
  const int per = n_heads / kv_heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = seq_slot[t];
  const int p = positions[t];
  // the first visible key: the window's, or (chunk > 0) the first position of the query's own run of `chunk` positions
  const int lo = chunk > 0 ? p / chunk * chunk : (window > 0 ? max(0, p - window + 1) : 0);
  const int n_kept = window > 0 ? min(keep_first, lo) : 0;
  const int n_keys = n_kept + p - lo + 1;
  const int k0 = c * kChunkKeys;
  const size_t stride = (size_t)vd + 2;
  if (slot < 0 || k0 >= n_keys) {  // nothing here: a partial result that the merge passes over
    if ((int)threadIdx.x < per) {
      float* dst = part + (((size_t)t * n_heads + g * per + threadIdx.x) * n_chunks + c) * stride;
      dst[0] = -INFINITY;
      dst[1] = 0.f;
    }
    return;
  }
  const int k1 = min(n_keys, k0 + kChunkKeys);
  const int width = (n_heads + kv_heads) * hd + kv_heads * vd;
  const __nv_bfloat16* q = qkv + (size_t)t * width + (size_t)g * per * hd;
  for (int i = threadIdx.x; i < per * hd; i += 32 * kWarps) q_s[i / hd][i % hd] = __bfloat162float(__ldcg(q + i));
  __syncthreads();

  const int* my_pages = pages + (size_t)t * max_blocks;
  const int idx = k0 + warp * kWarpKeys + (lane >> 1);
  const int j = idx < n_kept ? idx : lo + idx - n_kept;
  const int page = idx < k1 ? my_pages[j / kPage] : -1;
  const bool valid = page >= 0;
  const size_t row = valid ? ((size_t)page * kv_heads + g) * kPage + (j % kPage) : 0;

  float sc[PER];
#pragma unroll
  for (int h = 0; h < PER; ++h) sc[h] = 0.f;
  if (valid) {
    const __nv_bfloat16* k = kc + row * hd;
    constexpr int kPieces = 8;
    // (head sizes are multiples of 8: rows of 16-byte pieces, of which the key's two lanes take every other one)
    for (int d0 = (lane & 1) * 8; d0 < hd; d0 += 16 * kPieces) {
      uint4 raw[kPieces];
#pragma unroll
      for (int u = 0; u < kPieces; ++u)
        raw[u] = d0 + 16 * u < hd ? *reinterpret_cast<const uint4*>(k + d0 + 16 * u) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
      for (int u = 0; u < kPieces; ++u) {
        const int d = d0 + 16 * u;
        if (d >= hd) break;
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw[u]);
        float kv[8];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = __bfloat1622float2(h2[i]);
          kv[2 * i] = f.x;
          kv[2 * i + 1] = f.y;
        }
#pragma unroll
        for (int h = 0; h < PER; ++h) {
          if (h < per) {
            const float4 qa = *reinterpret_cast<const float4*>(&q_s[h][d]), qb = *reinterpret_cast<const float4*>(&q_s[h][d + 4]);
            sc[h] = fmaf(qa.x, kv[0], fmaf(qa.y, kv[1], fmaf(qa.z, kv[2], fmaf(qa.w, kv[3], sc[h]))));
            sc[h] = fmaf(qb.x, kv[4], fmaf(qb.y, kv[5], fmaf(qb.z, kv[6], fmaf(qb.w, kv[7], sc[h]))));
          }
        }
      }
    }
  }
  float pj[PER];
#pragma unroll
  for (int h = 0; h < PER; ++h) {
    const float slope = slopes && h < per ? slopes[g * per + h] : 0.f;
    const float hs = head_scales && h < per ? scale * head_scales[g * per + h] : scale;
    sc[h] += __shfl_xor_sync(0xffffffffu, sc[h], 1);
    const float near = dist_bias && valid && h < per ? dist_bias[(size_t)(g * per + h) * n_dist + min(p - j, n_dist - 1)] : 0.f;
    const float s = valid ? sc[h] * hs - slope * (float)(p - j) + near : -INFINITY;
    const float m = warp_max(s);  // (the warp's first key is always there: m is finite)
    pj[h] = valid ? expf(s - m) : 0.f;
    const float l = 0.5f * warp_sum(pj[h]);     // (every key counts in two lanes)
    if (lane == 0) {
      m_s[warp][h] = m;
      l_s[warp][h] = l;
    }
  }
  float acc[PER][DPL];
#pragma unroll
  for (int h = 0; h < PER; ++h)
#pragma unroll
    for (int i = 0; i < DPL; ++i) acc[h][i] = 0.f;
  const int n_valid = min(kWarpKeys, k1 - (k0 + warp * kWarpKeys));  // <= 0: this warp has no keys
  const bool dims = lane * DPL < vd;
  constexpr int kRowsAhead = 8;
  for (int j0 = 0; j0 < n_valid; j0 += kRowsAhead) {
    unsigned raw[kRowsAhead][DPL == 4 ? 2 : 1];     // a lane's values of a row: DPL of two bytes
#pragma unroll
    for (int u = 0; u < kRowsAhead; ++u) {           // (a lane without a key has probability zero and no row)
      const unsigned long long r = __shfl_sync(0xffffffffu, (unsigned long long)row, 2 * (j0 + u));
      const int there = __shfl_sync(0xffffffffu, (int)valid, 2 * (j0 + u));
      raw[u][0] = 0u;
      if constexpr (DPL == 4) raw[u][1] = 0u;
      if (dims && there) {
        const __nv_bfloat16* vr = vc + r * vd + lane * DPL;
        if constexpr (DPL == 4) {
          const uint2 two = *reinterpret_cast<const uint2*>(vr);
          raw[u][0] = two.x, raw[u][1] = two.y;
        } else if constexpr (DPL == 2) {
          raw[u][0] = *reinterpret_cast<const unsigned*>(vr);
        } else {
          raw[u][0] = *reinterpret_cast<const unsigned short*>(vr);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < kRowsAhead; ++u) {
      float v[DPL];
#pragma unroll
      for (int i = 0; i < DPL; ++i)      // bfloat16 is the upper half of a float
        v[i] = __uint_as_float(i % 2 == 0 ? raw[u][i / 2] << 16 : raw[u][i / 2] & 0xffff0000u);
#pragma unroll
      for (int h = 0; h < PER; ++h) {
        const float pv = __shfl_sync(0xffffffffu, pj[h], 2 * (j0 + u));
#pragma unroll
        for (int i = 0; i < DPL; ++i) acc[h][i] = fmaf(pv, v[i], acc[h][i]);
      }
    }
  }
  if (n_valid <= 0 && lane == 0) {
#pragma unroll
    for (int h = 0; h < PER; ++h) {
      m_s[warp][h] = -INFINITY;
      l_s[warp][h] = 0.f;
    }
  }
#pragma unroll
  for (int h = 0; h < PER; ++h)
#pragma unroll
    for (int i = 0; i < DPL; ++i) acc_s[warp][h][lane * DPL + i] = acc[h][i];
  __syncthreads();
  // the warps' results as one: thread per (head, value dim)
  for (int e = threadIdx.x; e < per * vd; e += 32 * kWarps) {
    const int h = e / vd, d = e % vd;
    float m = -INFINITY;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) m = fmaxf(m, m_s[w][h]);
    float l = 0.f, a = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float f = m_s[w][h] == -INFINITY ? 0.f : expf(m_s[w][h] - m);
      l = fmaf(l_s[w][h], f, l);
      a = fmaf(acc_s[w][h][d], f, a);
    }
    float* dst = part + (((size_t)t * n_heads + g * per + h) * n_chunks + c) * stride;
    if (d == 0) {
      dst[0] = m;
      dst[1] = l;
    }
    dst[2 + d] = a;
  }
}

// grid (T * n_heads): out = sum_c e^(m_c - M) acc_c / sum_c e^(m_c - M) l_c, chunks in order
__global__ void decode_kept_merge_kernel(const float* __restrict__ part, __nv_bfloat16* __restrict__ out,
                                         const int* __restrict__ seq_slot, int n_heads, int vd, int n_chunks,
                                         const float* __restrict__ sinks) {
  const int item = blockIdx.x, t = item / n_heads;
  __nv_bfloat16* o = out + (size_t)item * vd;
  if (seq_slot[t] < 0) {
    for (int d = threadIdx.x; d < vd; d += blockDim.x) o[d] = __float2bfloat16_rn(0.f);
    return;
  }
  const size_t stride = (size_t)vd + 2;
  const float* src = part + (size_t)item * n_chunks * stride;
  const int lane = threadIdx.x & 31;
  // every warp for itself: a lane a chunk (32 at a time) for the maximum, then for the factors e^(m_c - M) and the sum
  float m = sinks ? sinks[item % n_heads] : -INFINITY;
  for (int c0 = 0; c0 < n_chunks; c0 += 32) m = fmaxf(m, warp_max(c0 + lane < n_chunks ? src[(c0 + lane) * stride] : -INFINITY));
  float l = sinks ? expf(sinks[item % n_heads] - m) : 0.f;
  constexpr int kDims = 1;               // value dims a thread (the launch has a thread a dim)
  float a[kDims];
#pragma unroll
  for (int e = 0; e < kDims; ++e) a[e] = 0.f;
  for (int c0 = 0; c0 < n_chunks; c0 += 32) {
    const bool mine = c0 + lane < n_chunks;
    const float mc = mine ? src[(c0 + lane) * stride] : -INFINITY;
    const float f = mc == -INFINITY ? 0.f : expf(mc - m);
    l += warp_sum(f == 0.f ? 0.f : src[(c0 + lane) * stride + 1] * f);
    const int count = min(32, n_chunks - c0);
#pragma unroll 4
    for (int c = 0; c < count; ++c) {
      const float fc = __shfl_sync(0xffffffffu, f, c);
      if (fc == 0.f) continue;           // (a chunk without keys left nothing there; the same for every lane)
#pragma unroll
      for (int e = 0; e < kDims; ++e) {
        const int d = threadIdx.x + e * blockDim.x;
        if (d < vd) a[e] = fmaf(src[(c0 + c) * stride + 2 + d], fc, a[e]);
      }
    }
  }
  const float inv = 1.0f / l;
#pragma unroll
  for (int e = 0; e < kDims; ++e) {
    const int d = threadIdx.x + e * blockDim.x;
    if (d < vd) o[d] = __float2bfloat16_rn(a[e] * inv);
  }
}

template <int PER, int DPL>
void launch_partial(dim3 grid, cudaStream_t stream, const void* qkv, const void* kc, const void* vc, float* part,
                    const int* positions, const int* seq_slot, const int* pages, int max_blocks, int n_heads,
                    int kv_heads, int hd, int vd, float scale, int window, int keep_first, int n_chunks, const float* slopes,
                    int chunk, const float* head_scales, const float* dist_bias, int n_dist) {
  launch_plain(decode_kept_partial_kernel<PER, DPL>, grid, dim3(32 * kWarps), 0, stream, (const __nv_bfloat16*)qkv,
             (const __nv_bfloat16*)kc, (const __nv_bfloat16*)vc, part, positions, seq_slot, pages, max_blocks, n_heads,
             kv_heads, hd, vd, scale, window, keep_first, n_chunks, slopes, chunk, head_scales,
             dist_bias, n_dist);
}

}  // namespace

// Floats of scratch that a call needs.
EMBER_API size_t ember_attention_decode_kept_scratch(int T, int n_heads, int vd, int max_keys) {
  const size_t n_chunks = (size_t)((max_keys + kChunkKeys - 1) / kChunkKeys);
  return (size_t)T * n_heads * n_chunks * ((size_t)vd + 2);
}

// One token per sequence (token t is sequence t of the step), their keys and values already in the cache.
// max_keys: the most keys any token of the call can see (the grid is sized by it; a captured graph serves every
// length up to it).  Returns 2, having launched nothing, for sizes this kernel has no instantiation for
// (more than 8 query heads a key/value head, values of more than 128 or of an odd size above 32, head sizes that
// are no multiples of 8 or above 256): the caller then takes the plain kernel.
EMBER_API int ember_attention_decode_biased(const void* qkv, const void* kc, const void* vc, void* out, float* scratch,
                                            const int* positions, const int* seq_slot, const int* pages, int max_blocks,
                                            int T, int n_heads, int kv_heads, int hd, int vd, float scale, int window,
                                            int keep_first, int max_keys, const float* slopes, const float* sinks,
                                            cudaStream_t stream);

EMBER_API int ember_attention_decode_kept(const void* qkv, const void* kc, const void* vc, void* out, float* scratch,
                                          const int* positions, const int* seq_slot, const int* pages, int max_blocks,
                                          int T, int n_heads, int kv_heads, int hd, int vd, float scale, int window,
                                          int keep_first, int max_keys, cudaStream_t stream) {
  return ember_attention_decode_biased(qkv, kc, vc, out, scratch, positions, seq_slot, pages, max_blocks, T, n_heads, kv_heads,
                                       hd, vd, scale, window, keep_first, max_keys, nullptr, nullptr, stream);
}

// The same with a distance penalty (slopes: float32 per query head, or null) and a sink in the softmax's denominator
// (sinks: float32 per query head, or null).
EMBER_API int ember_attention_decode_chunked(const void* qkv, const void* kc, const void* vc, void* out, float* scratch,
                                             const int* positions, const int* seq_slot, const int* pages, int max_blocks,
                                             int T, int n_heads, int kv_heads, int hd, int vd, float scale, int window,
                                             int keep_first, int max_keys, const float* slopes, const float* sinks, int chunk,
                                             const float* head_scales, const float* dist_bias, int n_dist, cudaStream_t stream);

EMBER_API int ember_attention_decode_biased(const void* qkv, const void* kc, const void* vc, void* out, float* scratch,
                                            const int* positions, const int* seq_slot, const int* pages, int max_blocks,
                                            int T, int n_heads, int kv_heads, int hd, int vd, float scale, int window,
                                            int keep_first, int max_keys, const float* slopes, const float* sinks,
                                            cudaStream_t stream) {
  return ember_attention_decode_chunked(qkv, kc, vc, out, scratch, positions, seq_slot, pages, max_blocks, T, n_heads, kv_heads,
                                        hd, vd, scale, window, keep_first, max_keys, slopes, sinks, 0, nullptr, nullptr, 0, stream);
}

// The same with sight limited to the query's own chunk (chunk > 0, in place of a window) and one more factor on the
// scores of every query head (head_scales: float32 per query head, or null).  dist_bias: float32 [heads, n_dist] or null:
// what a score gains by the distance to the key, distances from n_dist - 1 on taking the last column.
EMBER_API int ember_attention_decode_chunked(const void* qkv, const void* kc, const void* vc, void* out, float* scratch,
                                             const int* positions, const int* seq_slot, const int* pages, int max_blocks,
                                             int T, int n_heads, int kv_heads, int hd, int vd, float scale, int window,
                                             int keep_first, int max_keys, const float* slopes, const float* sinks, int chunk,
                                             const float* head_scales, const float* dist_bias, int n_dist, cudaStream_t stream) {
  EMBER_CHECK(chunk >= 0 && (chunk == 0 || (window == 0 && keep_first == 0)), "attention_decode_kept: chunk %d beside window %d",
              chunk, window);
  EMBER_CHECK(T > 0 && n_heads > 0 && kv_heads > 0 && max_blocks > 0 && max_keys > 0, "attention_decode_kept: bad sizes");
  EMBER_CHECK(n_heads % kv_heads == 0, "attention_decode_kept: %d heads are not a multiple of %d key/value heads", n_heads,
              kv_heads);
  EMBER_CHECK(window >= 0 && keep_first >= 0, "attention_decode_kept: window %d, kept first %d", window, keep_first);
  EMBER_CHECK(dist_bias == nullptr || n_dist > 0, "attention_decode_kept: a bias for %d distances", n_dist);
  const int per = n_heads / kv_heads;
  int dpl = 0;
  for (int cand = 1; cand <= 4; cand *= 2)
    if (!dpl && vd <= 32 * cand && vd % cand == 0) dpl = cand;
  if (per > 8 || !dpl || hd % 8 || hd > 256) return 2;
  EMBER_CHECK(kv_heads <= 65535 && T <= 65535, "attention_decode_kept: %d tokens x %d heads exceed one launch", T, kv_heads);
  const int n_chunks = (max_keys + kChunkKeys - 1) / kChunkKeys;
  const dim3 grid(n_chunks, kv_heads, T);
  const int per_up = per <= 1 ? 1 : per <= 2 ? 2 : per <= 4 ? 4 : 8;
#define EMBER_KEPT(PER, DPL)                                                                                              \
  launch_partial<PER, DPL>(grid, stream, qkv, kc, vc, scratch, positions, seq_slot, pages, max_blocks, n_heads, kv_heads, \
                           hd, vd, scale, window, keep_first, n_chunks, slopes, chunk, head_scales, dist_bias, n_dist)
#define EMBER_KEPT_PER(PER)          \
  do {                               \
    if (dpl == 1) EMBER_KEPT(PER, 1); \
    else if (dpl == 2) EMBER_KEPT(PER, 2); \
    else EMBER_KEPT(PER, 4);          \
  } while (0)
  if (per_up == 1) EMBER_KEPT_PER(1);
  else if (per_up == 2) EMBER_KEPT_PER(2);
  else if (per_up == 4) EMBER_KEPT_PER(4);
  else EMBER_KEPT_PER(8);
#undef EMBER_KEPT_PER
#undef EMBER_KEPT
  EMBER_LAUNCH_OK("attention_decode_kept");
  launch_plain(decode_kept_merge_kernel, dim3(T * n_heads), dim3(vd <= 32 ? 32 : (vd <= 64 ? 64 : 128)), 0, stream,
             (const float*)scratch, (__nv_bfloat16*)out, seq_slot, n_heads, vd, n_chunks, sinks);
  EMBER_LAUNCH_OK("attention_decode_kept (merge)");
  return 0;
}
