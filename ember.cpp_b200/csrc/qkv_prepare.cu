// What stands between the projection of q, k and v and the attention, in one launch: norms over a whole row or over every
// head, a rotation, a norm after the rotation, and the keys' and values' way into the cache.
//
// A block takes one token (and, where tokens are few, a part of its heads).  A warp takes a head at a time: its values go
// through shared memory in float32, so that nothing is rounded between the norms and the rotation; the token's
// angles are turned into cos and sin once for all heads.  Rounding to the compute type happens once, at the store.  Query
// heads are written to the rows that the attention reads; keys and values go straight into the pages of the cache.
// Values may be the keys as projected (before norm and rotation): v_col is then k_col.  A warp's sums depend on the
// head's size alone, so a row's result does not depend on the batch.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;
constexpr int kMaxHead = 256;

enum : int { kNormNone = 0, kNormRow = 1, kNormHead = 2 };

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float total = 0.f;
  for (int i = 0; i < kWarps; ++i) total += red[i];
  return total;
}

__device__ __forceinline__ void store_pair(float* dst, float a, float b) { *reinterpret_cast<float2*>(dst) = make_float2(a, b); }
__device__ __forceinline__ void store_pair(__nv_bfloat16* dst, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(a, b);
}

struct Prepare {
  int heads, kv_heads, hd, vd;     // kv_heads 0: queries alone (the keys and values are another layer's)
  int k_col, v_col;                // columns of the projection; q starts at 0
  int norm;                        // before the rotation: none, over the row of heads, or a head at a time
  int unit_after;                  // after the rotation: q and k heads divided by their root mean square
  int dims, interleaved;           // rotated dimensions of a head (0: none) and how they pair
  float magnitude, eps;
};

template <typename TIN, typename TOUT>
__global__ void __launch_bounds__(kThreads)
qkv_prepare_kernel(const TIN* __restrict__ in, long long in_stride, TOUT* __restrict__ out, long long out_stride,
                   TOUT* __restrict__ kc, TOUT* __restrict__ vc, const int* __restrict__ positions,
                   const int* __restrict__ token_seq, const int* __restrict__ seq_slot, const int* __restrict__ pages,
                   int max_blocks, const float* __restrict__ q_gain, const float* __restrict__ k_gain,
                   const float* __restrict__ freqs, const Prepare a) {
  __shared__ float red[kWarps];
  __shared__ float cs[kMaxHead / 2], sn[kMaxHead / 2];
  __shared__ float buf_s[kWarps][kMaxHead];
  const int t = blockIdx.x, s = token_seq[t];
  if (seq_slot[s] < 0) return;          // padding: the attention writes its own zeros
  const int p = positions[t];
  const TIN* row = in + (size_t)t * in_stride;
  for (int i = threadIdx.x; i < a.dims / 2; i += kThreads) {
    float sv, cv;
    sincosf((float)p * freqs[i], &sv, &cv);
    cs[i] = cv * a.magnitude;
    sn[i] = sv * a.magnitude;
  }
  float inv_q = 1.f, inv_k = 1.f;
  if (a.norm == kNormRow) {
    const int qw = a.heads * a.hd, kw = a.kv_heads * a.hd;
    float ss = 0.f;
    for (int i = threadIdx.x; i < qw; i += kThreads) {
      const float v = to_float(row[i]);
      ss = fmaf(v, v, ss);
    }
    inv_q = 1.0f / sqrtf(block_sum(ss, red) / (float)qw + a.eps);
    if (kw > 0) {
      ss = 0.f;
      for (int i = threadIdx.x; i < kw; i += kThreads) {
        const float v = to_float(row[a.k_col + i]);
        ss = fmaf(v, v, ss);
      }
      inv_k = 1.0f / sqrtf(block_sum(ss, red) / (float)kw + a.eps);
    }
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* buf = buf_s[warp];
  const int page = a.kv_heads > 0 ? pages[(size_t)s * max_blocks + p / kPage] : 0;
  const int total = a.heads + 2 * a.kv_heads;
  for (int it = blockIdx.y * kWarps + warp; it < total; it += gridDim.y * kWarps) {
    if (it >= a.heads + a.kv_heads) {      // a value head: as projected
      if (page < 0) continue;
      const int g = it - a.heads - a.kv_heads;
      const TIN* src = row + a.v_col + (size_t)g * a.vd;
      TOUT* dst = vc + (((size_t)page * a.kv_heads + g) * kPage + p % kPage) * a.vd;
      for (int i = lane; i < a.vd; i += 32) dst[i] = from_float<TOUT>(to_float(src[i]));
      continue;
    }
    const bool key = it >= a.heads;
    const int h = key ? it - a.heads : it;
    if (key && page < 0) continue;
    const TIN* src = row + (key ? a.k_col : 0) + (size_t)h * a.hd;
    const float* gain = key ? k_gain : q_gain;
    const float inv_row = key ? inv_k : inv_q;
    float ss = 0.f;
    for (int i = lane; i < a.hd; i += 32) {
      float v = to_float(src[i]);
      ss = fmaf(v, v, ss);
      if (a.norm == kNormRow) v = v * inv_row * (gain ? gain[h * a.hd + i] : 1.f);
      buf[i] = v;
    }
    if (a.norm == kNormHead) {
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.hd + a.eps);
      for (int i = lane; i < a.hd; i += 32) buf[i] = buf[i] * inv * (gain ? gain[i] : 1.f);
    }
    __syncwarp();
    if (a.dims > 0) {
      const int half = a.dims / 2;
      for (int i = lane; i < half; i += 32) {
        const int iu = a.interleaved ? 2 * i : i, iv = a.interleaved ? 2 * i + 1 : i + half;
        const float u = buf[iu], v = buf[iv];
        buf[iu] = u * cs[i] - v * sn[i];
        buf[iv] = v * cs[i] + u * sn[i];
      }
      __syncwarp();
    }
    float inv = 1.f;
    if (a.unit_after) {
      ss = 0.f;
      for (int i = lane; i < a.hd; i += 32) ss = fmaf(buf[i], buf[i], ss);
      inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.hd + a.eps);
    }
    TOUT* dst = key ? kc + (((size_t)page * a.kv_heads + h) * kPage + p % kPage) * a.hd : out + (size_t)t * out_stride + (size_t)h * a.hd;
    if ((a.hd | (int)(out_stride & 1)) % 2 == 0)
      for (int i = lane * 2; i < a.hd; i += 64) store_pair(dst + i, buf[i] * inv, buf[i + 1] * inv);
    else
      for (int i = lane; i < a.hd; i += 32) dst[i] = from_float<TOUT>(buf[i] * inv);
    __syncwarp();
  }
}

}  // namespace

// in [T, *]: q (heads x hd) from column 0, and with kv_heads > 0 k (kv_heads x hd) from k_col and v (kv_heads x vd) from
// v_col.  out: rows of out_stride values whose first heads x hd are written.  kc, vc: the cache's pages (kv_heads > 0).
// norm 0 none, 1 over the row (gains of the row's width), 2 a head at a time (gains of hd values); gains null: ones.
EMBER_API int ember_qkv_prepare(const void* in, long long in_stride, void* out, long long out_stride, void* kc, void* vc,
                                const int* positions, const int* token_seq, const int* seq_slot, const int* pages, int max_blocks,
                                int T, int heads, int kv_heads, int hd, int vd, int k_col, int v_col, int norm, const float* q_gain,
                                const float* k_gain, float eps, int unit_after, const float* freqs, float magnitude, int dims,
                                int interleaved, int in_dtype, int out_dtype, cudaStream_t stream) {
  EMBER_CHECK(T > 0 && heads > 0 && kv_heads >= 0 && hd > 0 && hd <= kMaxHead && vd > 0 && vd <= kMaxHead, "qkv_prepare: bad sizes");
  EMBER_CHECK(in_stride >= (long long)heads * hd && out_stride >= (long long)heads * hd, "qkv_prepare: rows too short for q");
  EMBER_CHECK(kv_heads == 0 || (k_col >= 0 && v_col >= 0 && in_stride >= (long long)k_col + (long long)kv_heads * hd &&
                                in_stride >= (long long)v_col + (long long)kv_heads * vd && kc != nullptr && vc != nullptr &&
                                pages != nullptr && max_blocks > 0),
              "qkv_prepare: the keys' or values' columns do not fit the rows, or no cache");
  EMBER_CHECK(dims >= 0 && dims % 2 == 0 && dims <= hd && (dims == 0 || freqs != nullptr), "qkv_prepare: %d rotated dimensions of %d",
              dims, hd);
  EMBER_CHECK(norm >= 0 && norm <= 2, "qkv_prepare: norm %d", norm);
  Prepare a;
  a.heads = heads, a.kv_heads = kv_heads, a.hd = hd, a.vd = vd, a.k_col = k_col, a.v_col = v_col, a.norm = norm;
  a.unit_after = unit_after, a.dims = dims, a.interleaved = interleaved, a.magnitude = magnitude, a.eps = eps;
  const int total = heads + 2 * kv_heads;
  const int split = T >= 256 ? 1 : (total + kWarps - 1) / kWarps;      // few tokens: a warp a head over several blocks
  const dim3 grid(T, split < 65535 ? split : 65535);
  cudaError_t e;
#define EMBER_PREP(TIN, TOUT)                                                                                                    \
  launch_plain(qkv_prepare_kernel<TIN, TOUT>, grid, dim3(kThreads), 0, stream, (const TIN*)in, in_stride, (TOUT*)out, out_stride, \
               (TOUT*)kc, (TOUT*)vc, positions, token_seq, seq_slot, pages, max_blocks, q_gain, k_gain, freqs, a)
  if (in_dtype == EMBER_F32 && out_dtype == EMBER_F32) e = EMBER_PREP(float, float);
  else if (in_dtype == EMBER_F32 && out_dtype == EMBER_BF16) e = EMBER_PREP(float, __nv_bfloat16);
  else if (in_dtype == EMBER_BF16 && out_dtype == EMBER_BF16) e = EMBER_PREP(__nv_bfloat16, __nv_bfloat16);
  else return ember_fail("qkv_prepare: element types %d -> %d", in_dtype, out_dtype);
#undef EMBER_PREP
  if (e != cudaSuccess) return ember_fail("qkv_prepare: %s", cudaGetErrorString(e));
  return 0;
}
