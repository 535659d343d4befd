// What stands between the projection of q, k and v and the attention, in one launch: norms over a whole row or over every
// head, a rotation, a norm after the rotation, and the keys' and values' way into the cache.
//
// A block takes one token (and, where tokens are few, a part of its heads).  A warp takes a head at a time: its values go
// through shared memory in float32, so that nothing is rounded between the norms and the rotation; the token's
// angles are turned into cos and sin once for all heads.  Rounding to the compute type happens once, at the store.  Query
// heads are written to the rows that the attention reads; keys and values go straight into the pages of the cache.
// Values may be the keys as projected (before norm and rotation): v_col is then k_col.  With `blend` the values become
// (1 - blend) * own + blend * another layer's of the same token.  Without query heads (heads 0) only keys and values are made.  A warp's sums depend on the
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

// W values (4 or 1) from or to memory
template <int W>
__device__ __forceinline__ void load_w(const float* p, float (&v)[W]) {
  if constexpr (W == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w;
  } else {
    v[0] = *p;
  }
}
template <int W>
__device__ __forceinline__ void load_w(const __nv_bfloat16* p, float (&v)[W]) {
  if constexpr (W == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = lo.x, v[1] = lo.y, v[2] = hi.x, v[3] = hi.y;
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int W>
__device__ __forceinline__ void store_w(float* p, const float (&v)[W]) {
  if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int W>
__device__ __forceinline__ void store_w(__nv_bfloat16* p, const float (&v)[W]) {
  if constexpr (W == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

struct Prepare {
  int heads, kv_heads, hd, vd;     // kv_heads 0: queries alone (the keys and values are another layer's)
  int k_col, v_col;                // columns of the projection; q starts at 0
  int norm;                        // before the rotation: none, over the row of heads, or a head at a time
  int unit_after;                  // after the rotation: q and k heads divided by their root mean square
  int dims, interleaved;           // rotated dimensions of a head (0: none) and how they pair
  float magnitude, eps;
  const void* other;               // the values that are blended in: kv_heads x vd a row, or null
  long long other_stride;
  int other_bf16;
  float blend;
};

// W values of token t's row of the blended-in values, from column c on, folded into v
template <int W>
__device__ __forceinline__ void blend_values(const Prepare& a, int t, int c, float (&v)[W]) {
  if (a.other == nullptr) return;
  float o[W];
  if (a.other_bf16) load_w<W>(static_cast<const __nv_bfloat16*>(a.other) + (size_t)t * a.other_stride + c, o);
  else load_w<W>(static_cast<const float*>(a.other) + (size_t)t * a.other_stride + c, o);
#pragma unroll
  for (int e = 0; e < W; ++e) v[e] = (1.0f - a.blend) * v[e] + a.blend * o[e];
}

// W = 4: head sizes, columns and row strides are multiples of 4 and every pointer lies on 16 bytes (8 for bfloat16)
template <typename TIN, typename TOUT, int W>
__global__ void __launch_bounds__(kThreads)
qkv_prepare_kernel(const TIN* __restrict__ in, long long in_stride, TOUT* __restrict__ out, long long out_stride,
                   TOUT* __restrict__ kc, TOUT* __restrict__ vc, const int* __restrict__ positions,
                   const int* __restrict__ token_seq, const int* __restrict__ seq_slot, const int* __restrict__ pages,
                   int max_blocks, const float* __restrict__ q_gain, const float* __restrict__ k_gain,
                   const float* __restrict__ freqs, const Prepare a) {
  __shared__ float red[kWarps];
  __shared__ float cs[kMaxHead / 2], sn[kMaxHead / 2];
  __shared__ __align__(16) float buf_s[kWarps][kMaxHead];
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
    for (int i = threadIdx.x * W; i < qw; i += kThreads * W) {
      float v[W];
      load_w<W>(row + i, v);
#pragma unroll
      for (int e = 0; e < W; ++e) ss = fmaf(v[e], v[e], ss);
    }
    inv_q = 1.0f / sqrtf(block_sum(ss, red) / (float)qw + a.eps);
    if (kw > 0) {
      ss = 0.f;
      for (int i = threadIdx.x * W; i < kw; i += kThreads * W) {
        float v[W];
        load_w<W>(row + a.k_col + i, v);
#pragma unroll
        for (int e = 0; e < W; ++e) ss = fmaf(v[e], v[e], ss);
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
    if (it >= a.heads + a.kv_heads) {      // a value head: as projected, or blended with another layer's
      if (page < 0) continue;
      const int g = it - a.heads - a.kv_heads;
      const TIN* src = row + a.v_col + (size_t)g * a.vd;
      TOUT* dst = vc + (((size_t)page * a.kv_heads + g) * kPage + p % kPage) * a.vd;
      for (int i = lane * W; i < a.vd; i += 32 * W) {
        float v[W];
        load_w<W>(src + i, v);
        blend_values<W>(a, t, g * a.vd + i, v);
        store_w<W>(dst + i, v);
      }
      continue;
    }
    const bool key = it >= a.heads;
    const int h = key ? it - a.heads : it;
    if (key && page < 0) continue;
    const TIN* src = row + (key ? a.k_col : 0) + (size_t)h * a.hd;
    const float* gain = key ? k_gain : q_gain;
    const float inv_row = key ? inv_k : inv_q;
    float ss = 0.f;
    for (int i = lane * W; i < a.hd; i += 32 * W) {
      float v[W], g[W];
      load_w<W>(src + i, v);
#pragma unroll
      for (int e = 0; e < W; ++e) ss = fmaf(v[e], v[e], ss), g[e] = 1.f;
      if (a.norm == kNormRow) {
        if (gain) load_w<W>(gain + h * a.hd + i, g);
#pragma unroll
        for (int e = 0; e < W; ++e) v[e] = v[e] * inv_row * g[e];
      }
      store_w<W>(buf + i, v);
    }
    if (a.norm == kNormHead) {      // (a lane reads back what it wrote)
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.hd + a.eps);
      for (int i = lane * W; i < a.hd; i += 32 * W) {
        float v[W], g[W];
        load_w<W>(buf + i, v);
#pragma unroll
        for (int e = 0; e < W; ++e) g[e] = 1.f;
        if (gain) load_w<W>(gain + i, g);
#pragma unroll
        for (int e = 0; e < W; ++e) v[e] = v[e] * inv * g[e];
        store_w<W>(buf + i, v);
      }
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
      for (int i = lane * W; i < a.hd; i += 32 * W) {
        float v[W];
        load_w<W>(buf + i, v);
#pragma unroll
        for (int e = 0; e < W; ++e) ss = fmaf(v[e], v[e], ss);
      }
      inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.hd + a.eps);
    }
    TOUT* dst = key ? kc + (((size_t)page * a.kv_heads + h) * kPage + p % kPage) * a.hd : out + (size_t)t * out_stride + (size_t)h * a.hd;
    for (int i = lane * W; i < a.hd; i += 32 * W) {
      float v[W];
      load_w<W>(buf + i, v);
#pragma unroll
      for (int e = 0; e < W; ++e) v[e] *= inv;
      store_w<W>(dst + i, v);
    }
    __syncwarp();
  }
}

// The same for head sizes up to 128 in whole groups of four: a warp asks for the values of up to kItems heads before it waits
// for anything else (the token's place, its angles, another warp's sums), so that a block waits for memory about once.
constexpr int kItems = 3;

template <typename TIN, typename TOUT>
__global__ void __launch_bounds__(kThreads, 4)
qkv_prepare_short_kernel(const TIN* __restrict__ in, long long in_stride, TOUT* __restrict__ out, long long out_stride,
                         TOUT* __restrict__ kc, TOUT* __restrict__ vc, const int* __restrict__ positions,
                         const int* __restrict__ token_seq, const int* __restrict__ seq_slot, const int* __restrict__ pages,
                         int max_blocks, const float* __restrict__ q_gain, const float* __restrict__ k_gain,
                         const float* __restrict__ freqs, const Prepare a) {
  __shared__ float red[2][kWarps];
  __shared__ float cs[64], sn[64];
  __shared__ __align__(16) float buf_s[kWarps][128];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, col = lane * 4;
  const TIN* row = in + (size_t)t * in_stride;
  const int n_qk = a.heads + a.kv_heads, total = n_qk + a.kv_heads;
  const int first = blockIdx.y * kWarps + warp, step = gridDim.y * kWarps;
  float v[kItems][4];
  auto fetch = [&](int from) {
#pragma unroll
    for (int j = 0; j < kItems; ++j) {
      const int it = from + j * step;
      v[j][0] = v[j][1] = v[j][2] = v[j][3] = 0.f;
      if (it >= total) continue;
      const TIN* src = it < a.heads ? row + (size_t)it * a.hd
                       : it < n_qk  ? row + a.k_col + (size_t)(it - a.heads) * a.hd
                                    : row + a.v_col + (size_t)(it - n_qk) * a.vd;
      if (col < (it < n_qk ? a.hd : a.vd)) load_w<4>(src + col, v[j]);
    }
  };
  fetch(first);
  const int s = token_seq[t], p = positions[t];
  const bool live = seq_slot[s] >= 0;          // (uniform over the block)
  if (!live) return;                           // padding: the attention writes its own zeros
  const int page = a.kv_heads > 0 ? pages[(size_t)s * max_blocks + p / kPage] : 0;
  for (int i = threadIdx.x; i < a.dims / 2; i += kThreads) {
    float sv, cv;
    sincosf((float)p * freqs[i], &sv, &cv);
    cs[i] = cv * a.magnitude;
    sn[i] = sv * a.magnitude;
  }
  float inv_q = 1.f, inv_k = 1.f;
  if (a.norm == kNormRow) {
    // every warp's share of both rows of heads, in the order of the heads whatever the launch's shape
    float sq = 0.f, sk = 0.f;
    const bool held = gridDim.y == 1 && n_qk <= kItems * kWarps;      // (then it holds them already)
    for (int j0 = 0, it = warp; it < n_qk; ++j0, it += kWarps) {
      float w[4] = {0.f, 0.f, 0.f, 0.f};
      if (held) {
#pragma unroll
        for (int j = 0; j < kItems; ++j)
          if (j == j0) w[0] = v[j][0], w[1] = v[j][1], w[2] = v[j][2], w[3] = v[j][3];
      } else if (col < a.hd) {
        load_w<4>(it < a.heads ? row + (size_t)it * a.hd + col : row + a.k_col + (size_t)(it - a.heads) * a.hd + col, w);
      }
      const float ss = fmaf(w[0], w[0], fmaf(w[1], w[1], fmaf(w[2], w[2], w[3] * w[3])));
      if (it < a.heads) sq += ss;
      else sk += ss;
    }
    sq = warp_sum(sq), sk = warp_sum(sk);
    if (lane == 0) red[0][warp] = sq, red[1][warp] = sk;
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < kWarps; ++i) sq += red[0][i], sk += red[1][i];
    inv_q = 1.0f / sqrtf(sq / (float)(a.heads * a.hd) + a.eps);
    if (a.kv_heads > 0) inv_k = 1.0f / sqrtf(sk / (float)(a.kv_heads * a.hd) + a.eps);
  } else {
    __syncthreads();
  }
  float* buf = buf_s[warp];
  const bool mine = col < a.hd;
  const size_t place = p % kPage;
  for (int from = first; from < total; from += kItems * step) {
    if (from != first) fetch(from);
#pragma unroll
    for (int j = 0; j < kItems; ++j) {
      const int it = from + j * step;
      if (it >= total) break;
      if (it >= n_qk) {      // a value head: as projected, or blended with another layer's
        if (col < a.vd) blend_values<4>(a, t, (it - n_qk) * a.vd + col, v[j]);
        if (page >= 0 && col < a.vd) store_w<4>(vc + (((size_t)page * a.kv_heads + it - n_qk) * kPage + place) * a.vd + col, v[j]);
        continue;
      }
      const bool key = it >= a.heads;
      const int h = key ? it - a.heads : it;
      const float* gain = key ? k_gain : q_gain;
      float f = 1.f, g[4] = {1.f, 1.f, 1.f, 1.f};
      if (a.norm == kNormRow) {
        f = key ? inv_k : inv_q;
        if (gain && mine) load_w<4>(gain + h * a.hd + col, g);
      } else if (a.norm == kNormHead) {
        const float ss = warp_sum(fmaf(v[j][0], v[j][0], fmaf(v[j][1], v[j][1], fmaf(v[j][2], v[j][2], v[j][3] * v[j][3]))));
        f = 1.0f / sqrtf(ss / (float)a.hd + a.eps);
        if (gain && mine) load_w<4>(gain + col, g);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) v[j][e] = v[j][e] * f * g[e];
      if (a.dims > 0) {
        if (a.interleaved) {      // both of a pair are this lane's
#pragma unroll
          for (int e = 0; e < 4; e += 2)
            if (col + e < a.dims) {
              const float u = v[j][e], w = v[j][e + 1], c = cs[(col + e) / 2], sv = sn[(col + e) / 2];
              v[j][e] = u * c - w * sv;
              v[j][e + 1] = w * c + u * sv;
            }
        } else {
          const int half = a.dims / 2;
          if (mine) store_w<4>(buf + col, v[j]);
          __syncwarp();
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = col + e;
            if (i < half) v[j][e] = v[j][e] * cs[i] - buf[i + half] * sn[i];
            else if (i < a.dims) v[j][e] = v[j][e] * cs[i - half] + buf[i - half] * sn[i - half];
          }
          __syncwarp();
        }
      }
      if (a.unit_after) {
        const float ss = warp_sum(fmaf(v[j][0], v[j][0], fmaf(v[j][1], v[j][1], fmaf(v[j][2], v[j][2], v[j][3] * v[j][3]))));
        const float inv = 1.0f / sqrtf(ss / (float)a.hd + a.eps);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[j][e] *= inv;
      }
      if (!mine || (key && page < 0)) continue;
      store_w<4>(key ? kc + (((size_t)page * a.kv_heads + h) * kPage + place) * a.hd + col
                     : out + (size_t)t * out_stride + (size_t)h * a.hd + col, v[j]);
    }
  }
}

}  // namespace

// in [T, *]: q (heads x hd) from column 0, and with kv_heads > 0 k (kv_heads x hd) from k_col and v (kv_heads x vd) from
// v_col.  out: rows of out_stride values whose first heads x hd are written.  kc, vc: the cache's pages (kv_heads > 0).
// heads 0 (norm 0 or 2): keys and values alone, out is not touched.  other (float32 or bfloat16 rows of kv_heads x vd, or null):
// the values become (1 - blend) * own + blend * other.
// norm 0 none, 1 over the row (gains of the row's width), 2 a head at a time (gains of hd values); gains null: ones.
EMBER_API int ember_qkv_prepare(const void* in, long long in_stride, void* out, long long out_stride, void* kc, void* vc,
                                const int* positions, const int* token_seq, const int* seq_slot, const int* pages, int max_blocks,
                                int T, int heads, int kv_heads, int hd, int vd, int k_col, int v_col, int norm, const float* q_gain,
                                const float* k_gain, float eps, int unit_after, const float* freqs, float magnitude, int dims,
                                int interleaved, const void* other, long long other_stride, int other_dtype, float blend, int in_dtype, int out_dtype, cudaStream_t stream) {
  EMBER_CHECK(T > 0 && heads >= 0 && kv_heads >= 0 && heads + kv_heads > 0 && (heads > 0 || norm != kNormRow) && hd > 0 && hd <= kMaxHead && vd > 0 && vd <= kMaxHead, "qkv_prepare: bad sizes");
  EMBER_CHECK(in_stride >= (long long)heads * hd && out_stride >= (long long)heads * hd, "qkv_prepare: rows too short for q");
  EMBER_CHECK(kv_heads == 0 || (k_col >= 0 && v_col >= 0 && in_stride >= (long long)k_col + (long long)kv_heads * hd &&
                                in_stride >= (long long)v_col + (long long)kv_heads * vd && kc != nullptr && vc != nullptr &&
                                pages != nullptr && max_blocks > 0),
              "qkv_prepare: the keys' or values' columns do not fit the rows, or no cache");
  EMBER_CHECK(dims >= 0 && dims % 2 == 0 && dims <= hd && (dims == 0 || freqs != nullptr), "qkv_prepare: %d rotated dimensions of %d",
              dims, hd);
  EMBER_CHECK(other == nullptr || (kv_heads > 0 && other_stride >= (long long)kv_heads * vd && (other_dtype == EMBER_F32 || other_dtype == EMBER_BF16)),
              "qkv_prepare: the values to blend in do not fit");
  EMBER_CHECK(norm >= 0 && norm <= 2, "qkv_prepare: norm %d", norm);
  Prepare a;
  a.heads = heads, a.kv_heads = kv_heads, a.hd = hd, a.vd = vd, a.k_col = k_col, a.v_col = v_col, a.norm = norm;
  a.unit_after = unit_after, a.dims = dims, a.interleaved = interleaved, a.magnitude = magnitude, a.eps = eps;
  a.other = other, a.other_stride = other_stride, a.other_bf16 = other_dtype == EMBER_BF16, a.blend = blend;
  const int total = heads + 2 * kv_heads;
  const int split = T >= 256 ? 1 : (total + kWarps - 1) / kWarps;      // few tokens: a warp a head over several blocks
  const dim3 grid(T, split < 65535 ? split : 65535);
  cudaError_t e;
  const bool vec = (hd | vd | k_col | v_col) % 4 == 0 && in_stride % 4 == 0 && out_stride % 4 == 0 &&
                   (other == nullptr || (other_stride % 4 == 0 && (uintptr_t)other % (other_dtype == EMBER_BF16 ? 8 : 16) == 0)) &&
                   ((uintptr_t)in | (uintptr_t)out | (uintptr_t)kc | (uintptr_t)vc | (uintptr_t)q_gain | (uintptr_t)k_gain) % 16 == 0;
  const bool brief = vec && hd <= 128 && vd <= 128;
#define EMBER_PREP(TIN, TOUT)                                                                                                    \
  (brief ? launch_plain(qkv_prepare_short_kernel<TIN, TOUT>, grid, dim3(kThreads), 0, stream, (const TIN*)in, in_stride, (TOUT*)out, \
                        out_stride, (TOUT*)kc, (TOUT*)vc, positions, token_seq, seq_slot, pages, max_blocks, q_gain, k_gain, freqs, a) \
   : vec ? EMBER_PREP1(TIN, TOUT, 4) : EMBER_PREP1(TIN, TOUT, 1))
#define EMBER_PREP1(TIN, TOUT, W)                                                                                                \
  launch_plain(qkv_prepare_kernel<TIN, TOUT, W>, grid, dim3(kThreads), 0, stream, (const TIN*)in, in_stride, (TOUT*)out, out_stride, \
               (TOUT*)kc, (TOUT*)vc, positions, token_seq, seq_slot, pages, max_blocks, q_gain, k_gain, freqs, a)
  if (in_dtype == EMBER_F32 && out_dtype == EMBER_F32) e = EMBER_PREP(float, float);
  else if (in_dtype == EMBER_F32 && out_dtype == EMBER_BF16) e = EMBER_PREP(float, __nv_bfloat16);
  else if (in_dtype == EMBER_BF16 && out_dtype == EMBER_BF16) e = EMBER_PREP(__nv_bfloat16, __nv_bfloat16);
  else return ember_fail("qkv_prepare: element types %d -> %d", in_dtype, out_dtype);
#undef EMBER_PREP
#undef EMBER_PREP1
  if (e != cudaSuccess) return ember_fail("qkv_prepare: %s", cudaGetErrorString(e));
  return 0;
}
