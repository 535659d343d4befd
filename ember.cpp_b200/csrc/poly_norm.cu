// PolyNorm: a row activation of normed powers, for the inner rows of a feed-forward.
//
//   out = a N(z) + b N(z^2) + c N(z^3) + e,   N(v) = v / sqrt(mean(v^2) + eps) over the row
// (Zhuo et al., "Polynomial Composition Activations: Unleashing the Dynamics of Large Language Models").
//
// One block a row: the three sums of z^2, z^4 and z^6 in one pass, the result in a second; float32 arithmetic whatever
// the rows' element type.  A row's sums are added in an order that depends on its length alone.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x, v[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 raw;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = raw;
}

// VEC: rows are whole runs of 8 values on 16-byte boundaries
template <typename TIN, typename TOUT, bool VEC>
__global__ void __launch_bounds__(kThreads)
poly_norm_kernel(const TIN* __restrict__ in, TOUT* __restrict__ out, const float* __restrict__ four, int n, float eps) {
  __shared__ float red[3][kThreads / 32];
  const TIN* z = in + (size_t)blockIdx.x * n;
  TOUT* o = out + (size_t)blockIdx.x * n;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  auto add = [&](float v) {
    const float q = v * v, c = q * v;
    s1 += q;
    s2 = fmaf(q, q, s2);
    s3 = fmaf(c, c, s3);
  };
  if constexpr (VEC) {
    for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
      float v[8];
      load8(z + i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) add(v[e]);
    }
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) add(to_float(z[i]));
  }
  s1 = warp_sum(s1), s2 = warp_sum(s2), s3 = warp_sum(s3);
  if ((threadIdx.x & 31) == 0) {
    const int w = threadIdx.x >> 5;
    red[0][w] = s1, red[1][w] = s2, red[2][w] = s3;
  }
  __syncthreads();
  s1 = s2 = s3 = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) s1 += red[0][w], s2 += red[1][w], s3 += red[2][w];
  const float fa = four[0] / sqrtf(s1 / (float)n + eps), fb = four[1] / sqrtf(s2 / (float)n + eps),
              fc = four[2] / sqrtf(s3 / (float)n + eps), fe = four[3];
  auto result = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, fc, fb), fa), fe); };
  if constexpr (VEC) {
    for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
      float v[8];
      load8(z + i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = result(v[e]);
      store8(o + i, v);
    }
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) o[i] = from_float<TOUT>(result(to_float(z[i])));
  }
}

}  // namespace

// in, out [rows, n] (float32 -> float32 or bfloat16, bfloat16 -> bfloat16); four: a, b, c, e, float32 on the device
EMBER_API int ember_poly_norm(const void* in, void* out, const float* four, int rows, int n, float eps, int in_dtype, int out_dtype,
                              cudaStream_t stream) {
  EMBER_CHECK(rows > 0 && n > 0, "poly_norm: %d rows of %d", rows, n);
  const bool vec = n % 8 == 0 && ((uintptr_t)in | (uintptr_t)out) % 16 == 0;
  const int per = vec ? 8 : 1;
  const int threads = (n + per - 1) / per >= kThreads ? kThreads : ((n + per - 1) / per + 31) / 32 * 32;
  cudaError_t e;
#define EMBER_PN1(TIN, TOUT, VEC) \
  launch_plain(poly_norm_kernel<TIN, TOUT, VEC>, dim3(rows), dim3(threads), 0, stream, (const TIN*)in, (TOUT*)out, four, n, eps)
#define EMBER_PN(TIN, TOUT) (vec ? EMBER_PN1(TIN, TOUT, true) : EMBER_PN1(TIN, TOUT, false))
  if (in_dtype == EMBER_F32 && out_dtype == EMBER_F32) e = EMBER_PN(float, float);
  else if (in_dtype == EMBER_F32 && out_dtype == EMBER_BF16) e = EMBER_PN(float, __nv_bfloat16);
  else if (in_dtype == EMBER_BF16 && out_dtype == EMBER_BF16) e = EMBER_PN(__nv_bfloat16, __nv_bfloat16);
  else return ember_fail("poly_norm: element types %d -> %d", in_dtype, out_dtype);
#undef EMBER_PN
#undef EMBER_PN1
  if (e != cudaSuccess) return ember_fail("poly_norm: %s", cudaGetErrorString(e));
  return 0;
}
