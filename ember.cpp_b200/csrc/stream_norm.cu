// Arrangements whose norm comes after the sum, and layers whose output is a weighted sum over all layers in front.
//
//   post_norm       y = unit(alpha * x + sum_k f_k b_k) * (offset + w), the branches b_k with a factor each, with one
//                   more factor a row (an expert's weight) and with an RMS norm and gain of their own where they have them
//   with a history  X = y is a layer's result and the stream goes on as sum_j coef_j X_j + coef_n y over the results
//                   X_0 .. X_(n-1) of the layers in front (X_0: what the embedding left)
//   depth_average   that sum alone
//
// One block a row, float32 throughout; the row lies in shared memory between the sum and the norm.  Beside the float32
// stream the launch writes the row once more in the compute type, which is what the next sublayer's products read.
// A row is summed in an order that depends on its width alone.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;
constexpr int kMaxBranches = 32;
constexpr int kMaxHistory = 192;

struct Branches {
  const float* rows[kMaxBranches];
  long long stride[kMaxBranches];      // elements between two rows
  float factor[kMaxBranches];
  const float* weight[kMaxBranches];   // one more factor a row, weight[row * weight_stride], or null
  int weight_stride[kMaxBranches];
  const float* gain[kMaxBranches];     // the branch's own norm: divided by its root mean square, times this; null: as it is
  int n;
};

struct History {
  const float* x[kMaxHistory];
  int n;
};

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float total = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) total += red[i];
  return total;
}

// W values (4 or 1) at a time
template <int W>
struct Vals {
  float v[W];
};
template <int W>
__device__ __forceinline__ Vals<W> load_row(const float* p) {
  Vals<W> r;
  if constexpr (W == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    r.v[0] = a.x, r.v[1] = a.y, r.v[2] = a.z, r.v[3] = a.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int W>
__device__ __forceinline__ void store_row(float* p, const Vals<W>& r) {
  if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int W>
__device__ __forceinline__ void store_row(__nv_bfloat16* p, const Vals<W>& r) {
  if constexpr (W == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
    uint2 u;
    u.x = *reinterpret_cast<const unsigned*>(&lo);
    u.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
    *p = __float2bfloat16_rn(r.v[0]);
  }
}

template <int W>
__device__ __forceinline__ Vals<W> history_sum(const History& hist, const float* __restrict__ coef, size_t at) {
  Vals<W> a;
#pragma unroll
  for (int e = 0; e < W; ++e) a.v[e] = 0.f;
#pragma unroll 4
  for (int j = 0; j < hist.n; ++j) {
    const Vals<W> r = load_row<W>(hist.x[j] + at);
    const float c = coef[j];
#pragma unroll
    for (int e = 0; e < W; ++e) a.v[e] = fmaf(c, r.v[e], a.v[e]);
  }
  return a;
}

template <int W>
__global__ void __launch_bounds__(kThreads)
post_norm_kernel(const float* __restrict__ x, float alpha, const Branches b, const float* __restrict__ w, float offset, float eps,
                 float branch_eps, float* __restrict__ out, __nv_bfloat16* __restrict__ copy, const History hist,
                 const float* __restrict__ coef, float* __restrict__ mean, int d) {
  extern __shared__ __align__(16) float row_s[];
  __shared__ float red[kThreads / 32];
  __shared__ float f_s[kMaxBranches];
  const size_t row = blockIdx.x, base = row * (size_t)d;
  const int step = blockDim.x * W;
  if ((int)threadIdx.x < b.n) {
    const int k = threadIdx.x;
    f_s[k] = b.factor[k] * (b.weight[k] ? b.weight[k][row * (size_t)b.weight_stride[k]] : 1.f);
  }
  __syncthreads();
  for (int k = 0; k < b.n; ++k) {
    if (!b.gain[k]) continue;        // (uniform over the block)
    const float* r = b.rows[k] + row * (size_t)b.stride[k];
    float ss = 0.f;
    for (int i = threadIdx.x * W; i < d; i += step) {
      const Vals<W> v = load_row<W>(r + i);
#pragma unroll
      for (int e = 0; e < W; ++e) ss = fmaf(v.v[e], v.v[e], ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + branch_eps);
    if (threadIdx.x == 0) f_s[k] *= inv;
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x * W; i < d; i += step) {
    Vals<W> s = load_row<W>(x + base + i);
#pragma unroll
    for (int e = 0; e < W; ++e) s.v[e] *= alpha;
    for (int k = 0; k < b.n; ++k) {
      const Vals<W> v = load_row<W>(b.rows[k] + row * (size_t)b.stride[k] + i);
      const float f = f_s[k];
      if (b.gain[k]) {
        const Vals<W> g = load_row<W>(b.gain[k] + i);
#pragma unroll
        for (int e = 0; e < W; ++e) s.v[e] = fmaf(f * g.v[e], v.v[e], s.v[e]);
      } else {
#pragma unroll
        for (int e = 0; e < W; ++e) s.v[e] = fmaf(f, v.v[e], s.v[e]);
      }
    }
    store_row<W>(row_s + i, s);      // (read back by the same thread)
#pragma unroll
    for (int e = 0; e < W; ++e) ss = fmaf(s.v[e], s.v[e], ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
  const float c_last = mean ? coef[hist.n] : 0.f;
  for (int i = threadIdx.x * W; i < d; i += step) {
    Vals<W> y = load_row<W>(row_s + i);
    const Vals<W> g = load_row<W>(w + i);
#pragma unroll
    for (int e = 0; e < W; ++e) y.v[e] = y.v[e] * inv * (offset + g.v[e]);
    store_row<W>(out + base + i, y);
    if (mean) {
      Vals<W> a = history_sum<W>(hist, coef, base + i);
#pragma unroll
      for (int e = 0; e < W; ++e) y.v[e] = fmaf(c_last, y.v[e], a.v[e]);
      store_row<W>(mean + base + i, y);
    }
    if (copy) store_row<W>(copy + base + i, y);
  }
}

// The same for rows of up to 4 x blockDim.x values and NB branches or fewer: every thread has four values of each tensor
// in registers and asks for all of them before the first sum, so that a launch of few rows waits for memory once.
template <int NB>
__global__ void __launch_bounds__(1024)
post_norm_short_kernel(const float* __restrict__ x, float alpha, const Branches b, const float* __restrict__ w, float offset,
                       float eps, float branch_eps, float* __restrict__ out, __nv_bfloat16* __restrict__ copy, const History hist,
                       const float* __restrict__ coef, float* __restrict__ mean, int d) {
  __shared__ float red[NB + 1][32];
  const size_t row = blockIdx.x, base = row * (size_t)d;
  const int i = threadIdx.x * 4, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const bool there = i < d;
  const Vals<4> zero = {{0.f, 0.f, 0.f, 0.f}};
  Vals<4> s = zero, g = zero, a = zero, v[NB], bg[NB];
  float f[NB], c_last = 0.f;
  bool normed = false;
#pragma unroll
  for (int k = 0; k < NB; ++k) {
    v[k] = bg[k] = zero;
    f[k] = 0.f;
    if (k < b.n) {
      if (there) v[k] = load_row<4>(b.rows[k] + row * (size_t)b.stride[k] + i);
      if (there && b.gain[k]) bg[k] = load_row<4>(b.gain[k] + i);
      f[k] = b.factor[k] * (b.weight[k] ? b.weight[k][row * (size_t)b.weight_stride[k]] : 1.f);
      normed = normed || b.gain[k];
    }
  }
  if (there) {
    s = load_row<4>(x + base + i);
    g = load_row<4>(w + i);
    if (mean) {
      a = history_sum<4>(hist, coef, base + i);
      c_last = coef[hist.n];
    }
  }
  if (normed) {        // (uniform over the block)
#pragma unroll
    for (int k = 0; k < NB; ++k) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) ss = fmaf(v[k].v[e], v[k].v[e], ss);
      ss = warp_sum(ss);
      if (lane == 0) red[k][warp] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < NB; ++k) {
      if (k >= b.n || !b.gain[k]) continue;
      float total = 0.f;
      for (int q = 0; q < warps; ++q) total += red[k][q];
      f[k] *= 1.0f / sqrtf(total / (float)d + branch_eps);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    float t = alpha * s.v[e];
#pragma unroll
    for (int k = 0; k < NB; ++k)
      if (k < b.n) t = fmaf(b.gain[k] ? f[k] * bg[k].v[e] : f[k], v[k].v[e], t);
    s.v[e] = t;
    ss = fmaf(t, t, ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[NB][warp] = ss;
  __syncthreads();
  float total = 0.f;
  for (int q = 0; q < warps; ++q) total += red[NB][q];
  const float inv = 1.0f / sqrtf(total / (float)d + eps);
  if (!there) return;
#pragma unroll
  for (int e = 0; e < 4; ++e) s.v[e] = s.v[e] * inv * (offset + g.v[e]);
  store_row<4>(out + base + i, s);
  if (mean) {
#pragma unroll
    for (int e = 0; e < 4; ++e) s.v[e] = fmaf(c_last, s.v[e], a.v[e]);
    store_row<4>(mean + base + i, s);
  }
  if (copy) store_row<4>(copy + base + i, s);
}

template <int W>
__global__ void __launch_bounds__(kThreads)
depth_average_kernel(const History hist, const float* __restrict__ coef, float* __restrict__ mean, __nv_bfloat16* __restrict__ copy,
                     size_t total) {
  const size_t step = (size_t)gridDim.x * blockDim.x * W;
  for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * W; i < total; i += step) {
    const Vals<W> a = history_sum<W>(hist, coef, i);
    store_row<W>(mean + i, a);
    if (copy) store_row<W>(copy + i, a);
  }
}

int fill_history(History& h, const void* const* rows, int n, bool& vec) {
  if (n < 0 || n > kMaxHistory) return ember_fail("depth average: %d layers in front (at most %d)", n, kMaxHistory);
  h.n = n;
  for (int j = 0; j < n; ++j) {
    h.x[j] = (const float*)rows[j];
    vec = vec && (uintptr_t)rows[j] % 16 == 0;
  }
  return 0;
}

}  // namespace

// x, out, mean float32 [rows, d]; copy bfloat16 [rows, d] or null (of `mean` where there is one, else of `out`).
// Host arrays of n_branches entries: rows (float32), strides (elements), factors, weights (device pointers or null) with
// weight_strides, gains (device pointers or null).  history: host array of n_history float32 [rows, d] tensors, coef
// float32 [n_history + 1] on the device, mean: all three or none (mean null).
EMBER_API int ember_post_norm(const float* x, float alpha, const void* const* rows, const long long* strides, const float* factors,
                              const void* const* weights, const int* weight_strides, const void* const* gains, int n_branches,
                              const float* w, float offset, float eps, float branch_eps, float* out, void* copy,
                              const void* const* history, int n_history, const float* coef, float* mean, int n_rows, int d,
                              cudaStream_t stream) {
  EMBER_CHECK(n_rows > 0 && d > 0 && d <= 12000, "post_norm: %d rows of %d (at most 12000)", n_rows, d);
  EMBER_CHECK(n_branches >= 1 && n_branches <= kMaxBranches, "post_norm: %d branches (1 to %d)", n_branches, kMaxBranches);
  EMBER_CHECK(mean == nullptr || coef != nullptr, "post_norm: an average without coefficients");
  bool vec = d % 4 == 0 && ((uintptr_t)x | (uintptr_t)w | (uintptr_t)out | (uintptr_t)mean) % 16 == 0 && (uintptr_t)copy % 8 == 0;
  Branches b = {};
  b.n = n_branches;
  for (int k = 0; k < n_branches; ++k) {
    b.rows[k] = (const float*)rows[k];
    b.stride[k] = strides[k];
    b.factor[k] = factors[k];
    b.weight[k] = (const float*)weights[k];
    b.weight_stride[k] = weight_strides[k];
    b.gain[k] = (const float*)gains[k];
    vec = vec && strides[k] % 4 == 0 && ((uintptr_t)rows[k] | (uintptr_t)gains[k]) % 16 == 0;
  }
  History h = {};
  if (mean != nullptr && fill_history(h, history, n_history, vec)) return 1;
  const int per = vec ? 4 : 1;
  const int threads = (d + per - 1) / per >= kThreads ? kThreads : ((d + per - 1) / per + 31) / 32 * 32;
  const size_t smem = (size_t)d * sizeof(float);
  // (2,048 rows of 2,048: 26 microseconds a launch with the loop, 30 with the registers; 8 rows: 17 and 14.  Without a copy
  // the stream is the compute type's own, float32: one kernel whatever the rows, so that every cut of the work adds alike)
  if (vec && copy != nullptr && n_rows < 512 && d <= 4096 && n_branches <= 4) {
    const int quads = (d / 4 + 31) / 32 * 32;
#define EMBER_PN(NB)                                                                                                               \
  launch_plain(post_norm_short_kernel<NB>, dim3(n_rows), dim3(quads), 0, stream, x, alpha, b, w, offset, eps, branch_eps, out, \
               (__nv_bfloat16*)copy, h, coef, mean, d)
    const cudaError_t e = n_branches == 1 ? EMBER_PN(1) : n_branches == 2 ? EMBER_PN(2) : EMBER_PN(4);
#undef EMBER_PN
    if (e != cudaSuccess) return ember_fail("post_norm: %s", cudaGetErrorString(e));
    return 0;
  }
  const cudaError_t e =
      vec ? launch_plain(post_norm_kernel<4>, dim3(n_rows), dim3(threads), smem, stream, x, alpha, b, w, offset, eps, branch_eps, out,
                         (__nv_bfloat16*)copy, h, coef, mean, d)
          : launch_plain(post_norm_kernel<1>, dim3(n_rows), dim3(threads), smem, stream, x, alpha, b, w, offset, eps, branch_eps, out,
                         (__nv_bfloat16*)copy, h, coef, mean, d);
  if (e != cudaSuccess) return ember_fail("post_norm: %s", cudaGetErrorString(e));
  return 0;
}

// mean = sum over j < n of coef[j] * history[j] (float32 [total] each), copy: the same in bfloat16, or null
EMBER_API int ember_depth_average(const void* const* history, int n_history, const float* coef, float* mean, void* copy, size_t total,
                                  cudaStream_t stream) {
  EMBER_CHECK(total > 0 && n_history > 0, "depth_average: %d tensors", n_history);
  bool vec = total % 4 == 0 && (uintptr_t)mean % 16 == 0 && (uintptr_t)copy % 8 == 0;
  History h = {};
  if (fill_history(h, history, n_history, vec)) return 1;
  const size_t items = vec ? total / 4 : total;
  const int grid = (int)((items + kThreads - 1) / kThreads < 65535 ? (items + kThreads - 1) / kThreads : 65535);
  const cudaError_t e = vec ? launch_plain(depth_average_kernel<4>, dim3(grid), dim3(kThreads), 0, stream, h, coef, mean,
                                           (__nv_bfloat16*)copy, total)
                            : launch_plain(depth_average_kernel<1>, dim3(grid), dim3(kThreads), 0, stream, h, coef, mean,
                                           (__nv_bfloat16*)copy, total);
  if (e != cudaSuccess) return ember_fail("depth_average: %s", cudaGetErrorString(e));
  return 0;
}
