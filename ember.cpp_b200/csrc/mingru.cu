// minGRU over a step's packed tokens: a recurrence per channel whose gates read the current token alone.
//
//     z_t = sigmoid(a_t + bias_z)      u_t = b_t + bias_x      c_t = u_t + 1/2 where u_t >= 0, sigmoid(u_t) where u_t < 0
//     S_t = (1 - z_t) S_(t-1) + z_t c_t                         out_t = S_t * silu(g_t)
// a, b and g are columns of one projection (the step's rows of z | x | g).  Gates, candidates and the state
// are float32 whatever the element types that come in or go out.  The walk is channel_scan.cuh's.
#include "channel_scan.cuh"

namespace {

__device__ __forceinline__ float sigmoidf(float v) { return 1.0f / (1.0f + expf(-v)); }

template <typename TIN>
struct MinGru {
  const TIN* proj;
  long long stride;
  int z_col, x_col, g_col;
  const float *bias_z, *bias_x;
  float bz, bx;
  struct Row {
    float z, x, g;
  };
  __device__ __forceinline__ void begin(int c) {
    bz = bias_z[c];
    bx = bias_x[c];
  }
  __device__ __forceinline__ Row fetch(size_t t, int c, int phase) const {
    const TIN* row = proj + t * stride;
    return Row{to_float(row[z_col + c]), to_float(row[x_col + c]), phase != 1 ? to_float(row[g_col + c]) : 0.f};
  }
  __device__ __forceinline__ void keep(size_t, int, float, float) const {}
  __device__ __forceinline__ void factors(const Row& r, int, float& A, float& B) const {
    const float z = sigmoidf(r.z + bz), b = r.x + bx;
    A = 1.0f - z;
    B = z * (b >= 0.f ? b + 0.5f : sigmoidf(b));
  }
  __device__ __forceinline__ float result(const Row& r, float S) const { return S * (r.g * sigmoidf(r.g)); }
};

}  // namespace

EMBER_API size_t ember_mingru_scratch(int n_seqs, int pieces, int width) { return scan::scratch_floats(n_seqs, pieces, width); }

// proj: rows of `stride` values with the gate's, the candidate's and the output gate's `width` columns from z_col, x_col
// and g_col; biases float32 [width]; state float32 [slots, width] (advanced); out [T, width].  pieces 1: one walk;
// more (with scratch of ember_mingru_scratch floats): pieces of `piece` tokens side by side.
EMBER_API int ember_mingru(const void* proj, long long stride, int z_col, int x_col, int g_col, const float* bias_z,
                           const float* bias_x, float* state, void* out, const int* seq_slot, const int* seq_start,
                           const int* cu_new, int n_seqs, int width, int piece, int pieces, float* scratch, int in_dtype,
                           int out_dtype, cudaStream_t stream) {
  EMBER_CHECK(n_seqs > 0 && width > 0 && pieces >= 1 && piece >= 1, "mingru: bad sizes");
  EMBER_CHECK(pieces == 1 || scratch != nullptr, "mingru: pieces side by side need scratch");
  EMBER_CHECK(pieces <= 65535, "mingru: %d pieces exceed one launch", pieces);
  EMBER_CHECK((in_dtype == EMBER_F32 || in_dtype == EMBER_BF16) && (out_dtype == EMBER_F32 || out_dtype == EMBER_BF16) &&
                  !(in_dtype == EMBER_BF16 && out_dtype == EMBER_F32),
              "mingru: element types %d -> %d", in_dtype, out_dtype);
#define EMBER_GRU(TIN, TOUT)                                                                                                  \
  scan::launch(MinGru<TIN>{(const TIN*)proj, stride, z_col, x_col, g_col, bias_z, bias_x, 0.f, 0.f}, state, (TOUT*)out, seq_slot, \
               seq_start, cu_new, n_seqs, width, piece, pieces, scratch, stream)
  const cudaError_t e = in_dtype == EMBER_BF16    ? EMBER_GRU(__nv_bfloat16, __nv_bfloat16)
                        : out_dtype == EMBER_BF16 ? EMBER_GRU(float, __nv_bfloat16)
                                                  : EMBER_GRU(float, float);
#undef EMBER_GRU
  if (e != cudaSuccess) return ember_fail("mingru: %s", cudaGetErrorString(e));
  return 0;
}
