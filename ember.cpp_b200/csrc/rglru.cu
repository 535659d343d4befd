// The real-gated linear recurrent unit over a step's packed tokens (De et al., "Griffin: Mixing Gated Linear Recurrences
// with Local Attention for Efficient Language Models"): a recurrence per channel with a decay between zero and one.
//
//     r_t = sigmoid(zr_t + bias_r)      i_t = sigmoid(zi_t + bias_i)      log a_t = -rate * r_t      a_t = exp(log a_t)
//     S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t                         out_t = S_t * gelu_tanh(y_t)
// rate >= 0 is a constant of the channel (a factor times softplus of a learned number).  zr and zi are products of u with
// a square matrix for each of `parts` equal parts of the channels: rows of 2 * width values in which part b holds its
// n = width / parts values of zr, then its n values of zi.  Everything from the products on is float32.  With
// m = exp(log a) - 1 (one expm1), a = 1 + m and 1 - a^2 = -m (2 + m), exact where a is close to one.
//
//   ember_rglru       the recurrence over rows of zr | zi (the walk is channel_scan.cuh's; where pieces are walked twice, the
//                     first walk leaves a and sqrt(1 - a^2) i u in the places of zr and zi for the second)
//   ember_rglru_step  steps that bring one token a sequence: the products of the gates and the recurrence in one launch;
//                     a warp makes both gates of a channel for eight sequences, so that a matrix row is read once for them
#include "channel_scan.cuh"

namespace {

__device__ __forceinline__ float sigmoidf(float v) { return __fdividef(1.0f, 1.0f + expf(-v)); }
// the tanh form of GELU, 0.5 (1 + tanh(x)) being sigmoid(2 x)
__device__ __forceinline__ float gelu_gate(float v) { return v * sigmoidf(1.5957691216057308f * (v + 0.044715f * v * v * v)); }

__device__ __forceinline__ void rglru_factors(float zr, float zi, float u, float rate, float& A, float& B) {
  const float m = expm1f(-rate * sigmoidf(zr));
  A = 1.0f + m;
  B = sqrtf(-m * (2.0f + m)) * sigmoidf(zi) * u;      // (-1 <= m <= 0)
}

template <typename T>
struct RgLru {
  float* gates;             // [T, 2 * width]
  const T* u;               // [T, width]
  const T* y;               // rows of y_stride values, the channel's value at column c
  long long y_stride;
  const float *bias_r, *bias_i, *rate;
  int width, part;
  float br, bi, rt;
  int col;
  struct Row {
    float zr, zi, u, y;
  };
  __device__ __forceinline__ void begin(int c) {
    br = bias_r[c];
    bi = bias_i[c];
    rt = rate[c];
    col = c / part * 2 * part + c % part;
  }
  __device__ __forceinline__ Row fetch(size_t t, int c, int phase) const {
    const float* g = gates + t * 2 * width + col;
    return Row{g[0], g[part], phase != 2 ? to_float(u[t * width + c]) : 0.f, phase != 1 ? to_float(y[t * y_stride + c]) : 0.f};
  }
  __device__ __forceinline__ void factors(const Row& r, int phase, float& A, float& B) const {
    if (phase == 2) A = r.zr, B = r.zi;
    else rglru_factors(r.zr + br, r.zi + bi, r.u, rt, A, B);
  }
  __device__ __forceinline__ void keep(size_t t, int, float A, float B) const {
    float* g = gates + t * 2 * width + col;
    g[0] = A;
    g[part] = B;
  }
  __device__ __forceinline__ float result(const Row& r, float S) const { return S * gelu_gate(r.y); }
};

constexpr int kStepWarps = 8;
constexpr int kStepSeqs = 8;      // sequences that share a read of a matrix row

// grid (channels of a part / kStepWarps, parts, sequences / kStepSeqs); token t of the step is sequence t.  Dynamic shared
// memory: kStepSeqs rows of n values of u (float32).
__global__ void __launch_bounds__(32 * kStepWarps)
rglru_step_kernel(const __nv_bfloat16* __restrict__ u, const __nv_bfloat16* __restrict__ y, long long y_stride,
                  const __nv_bfloat16* __restrict__ w, const float* __restrict__ bias_r, const float* __restrict__ bias_i,
                  const float* __restrict__ rate, float* __restrict__ state, __nv_bfloat16* __restrict__ out,
                  const int* __restrict__ seq_slot, const int* __restrict__ seq_start, int T, int width, int n) {
  extern __shared__ __align__(16) float u_s[];
  const int b = blockIdx.y, t0 = blockIdx.z * kStepSeqs, count = min(kStepSeqs, T - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < kStepSeqs * n; i += 32 * kStepWarps) {
    const int s = i / n;
    u_s[i] = s < count ? __bfloat162float(u[(size_t)(t0 + s) * width + (size_t)b * n + i % n]) : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.x * kStepWarps + warp;
  if (c >= n) return;
  const __nv_bfloat16* wr = w + ((size_t)b * 2 * n + c) * n;       // part b: n rows of the first gate, then n of the second
  const __nv_bfloat16* wi = wr + (size_t)n * n;
  float ar[kStepSeqs], ai[kStepSeqs];
#pragma unroll
  for (int s = 0; s < kStepSeqs; ++s) ar[s] = ai[s] = 0.f;
  for (int k = lane * 2; k < n; k += 64) {      // (n is even: rows of whole pairs)
    const float2 fr = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(wr + k));
    const float2 fi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(wi + k));
#pragma unroll
    for (int s = 0; s < kStepSeqs; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(u_s + s * n + k);
      ar[s] = fmaf(fr.x, v.x, fmaf(fr.y, v.y, ar[s]));
      ai[s] = fmaf(fi.x, v.x, fmaf(fi.y, v.y, ai[s]));
    }
  }
  float zr = 0.f, zi = 0.f;
#pragma unroll
  for (int s = 0; s < kStepSeqs; ++s) {
    const float r = warp_sum(ar[s]), i = warp_sum(ai[s]);
    if (lane == s) zr = r, zi = i;
  }
  if (lane >= count) return;
  const int t = t0 + lane, ch = b * n + c, slot = seq_slot[t];
  __nv_bfloat16* o = out + (size_t)t * width + ch;
  if (slot < 0) {
    *o = __float2bfloat16_rn(0.f);
    return;
  }
  float A, B;
  rglru_factors(zr + bias_r[ch], zi + bias_i[ch], u_s[lane * n + c], rate[ch], A, B);
  float* st = state + (size_t)slot * width + ch;
  const float S = fmaf(A, seq_start[t] > 0 ? *st : 0.f, B);
  *st = S;
  *o = __float2bfloat16_rn(S * gelu_gate(__bfloat162float(y[(size_t)t * y_stride + ch])));
}

}  // namespace

EMBER_API size_t ember_rglru_scratch(int n_seqs, int pieces, int width) { return scan::scratch_floats(n_seqs, pieces, width); }

// gates float32 [T, 2 * width] (see above; overwritten where pieces > 1), u [T, width] and y (rows of y_stride values) of one element type, biases and
// rate float32 [width], state float32 [slots, width] (advanced), out [T, width] of u's type.
EMBER_API int ember_rglru(float* gates, const void* u, const void* y, long long y_stride, const float* bias_r,
                          const float* bias_i, const float* rate, float* state, void* out, const int* seq_slot,
                          const int* seq_start, const int* cu_new, int n_seqs, int width, int parts, int piece, int pieces,
                          float* scratch, int dtype, cudaStream_t stream) {
  EMBER_CHECK(n_seqs > 0 && width > 0 && parts > 0 && width % parts == 0 && pieces >= 1 && piece >= 1, "rglru: bad sizes");
  EMBER_CHECK(pieces == 1 || scratch != nullptr, "rglru: pieces side by side need scratch");
  EMBER_CHECK(pieces <= 65535, "rglru: %d pieces exceed one launch", pieces);
#define EMBER_RG(T)                                                                                                            \
  scan::launch(RgLru<T>{gates, (const T*)u, (const T*)y, y_stride, bias_r, bias_i, rate, width, width / parts, 0.f, 0.f, 0.f, 0}, \
               state, (T*)out, seq_slot, seq_start, cu_new, n_seqs, width, piece, pieces, scratch, stream)
  cudaError_t e;
  if (dtype == EMBER_F32) e = EMBER_RG(float);
  else if (dtype == EMBER_BF16) e = EMBER_RG(__nv_bfloat16);
  else return ember_fail("rglru: element type %d", dtype);
#undef EMBER_RG
  if (e != cudaSuccess) return ember_fail("rglru: %s", cudaGetErrorString(e));
  return 0;
}

// One token a sequence (token t is sequence t), bfloat16: w [parts, 2 * n, n] with n = width / parts, the first gate's rows
// of a part, then the second's.  Returns 2, having launched nothing, where n is odd or above 1,024.
EMBER_API int ember_rglru_step(const void* u, const void* y, long long y_stride, const void* w, const float* bias_r,
                               const float* bias_i, const float* rate, float* state, void* out, const int* seq_slot,
                               const int* seq_start, int T, int width, int parts, cudaStream_t stream) {
  EMBER_CHECK(T > 0 && width > 0 && parts > 0 && width % parts == 0, "rglru_step: bad sizes");
  const int n = width / parts;
  if (n % 2 || n > 1024 || parts > 65535) return 2;
  const dim3 grid((n + kStepWarps - 1) / kStepWarps, parts, (T + kStepSeqs - 1) / kStepSeqs);
  const cudaError_t e = launch_plain(rglru_step_kernel, grid, dim3(32 * kStepWarps), (size_t)kStepSeqs * n * sizeof(float), stream,
                                     (const __nv_bfloat16*)u, (const __nv_bfloat16*)y, y_stride, (const __nv_bfloat16*)w, bias_r,
                                     bias_i, rate, state, (__nv_bfloat16*)out, seq_slot, seq_start, T, width, n);
  if (e != cudaSuccess) return ember_fail("rglru_step: %s", cudaGetErrorString(e));
  return 0;
}
