// A linear recurrence per channel over a step's packed tokens: S_t = A_t S_(t-1) + B_t, the factors read from the
// current token alone (a "rule" says how), the results a function of S_t and the token.
//
// A thread takes a channel through a sequence's tokens in order, so a token's result depends on its
// sequence alone.  A long sequence is cut into pieces that are walked side by side: a piece walked from zero gives
// (product of its A, its end value from zero); the pieces' start values follow from those in order, and a second walk
// from each piece's start value writes the results.  A sequence that starts at position 0 starts from zeros whatever its
// slot's state holds; sequences of slot -1 are padding: their rows are zero and no state is touched.
//
// A rule has
//   struct Row               the values of one token and channel, as fetched
//   begin(c)                 what a channel keeps (biases)
//   fetch(t, c, phase)       a token's Row for a phase (see the kernel: what a phase does not need may be left out)
//   factors(row, phase, A, B)  A_t and B_t
//   keep(t, c, A, B)         the first walk's factors, for a rule that leaves them to the second walk (or nothing)
//   result(row, S)           the token's output
#pragma once

#include "common.cuh"

namespace scan {

constexpr int kThreads = 128;

// grid (sequences, channel tiles, pieces).  phase 0: the whole walk (one piece).  phase 1: a piece from zero,
// leaving (product of A, end value) in scratch.  phase 2: the walk from the piece's start value, which the
// carry left in scratch.
template <int phase, typename Rule, typename TOUT>
__global__ void __launch_bounds__(kThreads)
channel_scan_kernel(Rule rule, float* __restrict__ state, TOUT* __restrict__ out, const int* __restrict__ seq_slot,
                    const int* __restrict__ seq_start, const int* __restrict__ cu_new, int width, int piece,
                    float* __restrict__ scratch) {
  const int s = blockIdx.x, c = blockIdx.y * kThreads + threadIdx.x, p = blockIdx.z;
  if (c >= width) return;
  const int t0 = cu_new[s], n = cu_new[s + 1] - t0;
  const int lo = p * piece, hi = min(n, lo + piece);
  const int slot = seq_slot[s];
  if (slot < 0) {
    if (phase != 1)
      for (int i = lo; i < hi; ++i) out[(size_t)(t0 + i) * width + c] = from_float<TOUT>(0.f);
    return;
  }
  if (lo >= n) return;
  rule.begin(c);
  float* mine = scratch ? scratch + (((size_t)s * gridDim.z + p) * width + c) * 2 : nullptr;
  float S = 0.f;
  if (phase == 0) S = seq_start[s] > 0 ? state[(size_t)slot * width + c] : 0.f;
  if (phase == 2) S = mine[1];
  float all = 1.f;
  constexpr int kAhead = 8;      // tokens whose columns are fetched, and whose factors are made, before the chain walks them
  int i0 = lo;
  for (; i0 + kAhead <= hi; i0 += kAhead) {
    typename Rule::Row rows[kAhead];
    float A[kAhead], B[kAhead];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) rows[u] = rule.fetch((size_t)(t0 + i0 + u), c, phase);
#pragma unroll
    for (int u = 0; u < kAhead; ++u) rule.factors(rows[u], phase, A[u], B[u]);
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      S = fmaf(A[u], S, B[u]);
      if (phase == 1) {
        all *= A[u];
        rule.keep((size_t)(t0 + i0 + u), c, A[u], B[u]);
      } else {
        out[(size_t)(t0 + i0 + u) * width + c] = from_float<TOUT>(rule.result(rows[u], S));
      }
    }
  }
  for (; i0 < hi; ++i0) {
    float A, B;
    const typename Rule::Row row = rule.fetch((size_t)(t0 + i0), c, phase);
    rule.factors(row, phase, A, B);
    S = fmaf(A, S, B);
    if (phase == 1) {
      all *= A;
      rule.keep((size_t)(t0 + i0), c, A, B);
    } else {
      out[(size_t)(t0 + i0) * width + c] = from_float<TOUT>(rule.result(row, S));
    }
  }
  if (phase == 1) {
    mine[0] = all;
    mine[1] = S;
  } else if (hi == n) {
    state[(size_t)slot * width + c] = S;
  }
}

// grid (sequences, channel tiles): scratch (product of A, end from zero) of every piece becomes (product, start value).
static __global__ void channel_carry_kernel(float* __restrict__ scratch, const float* __restrict__ state,
                                            const int* __restrict__ seq_slot, const int* __restrict__ seq_start,
                                            const int* __restrict__ cu_new, int width, int piece, int pieces) {
  const int s = blockIdx.x, c = blockIdx.y * kThreads + threadIdx.x;
  if (c >= width) return;
  const int slot = seq_slot[s];
  if (slot < 0) return;
  const int n = cu_new[s + 1] - cu_new[s];
  float S = seq_start[s] > 0 ? state[(size_t)slot * width + c] : 0.f;
  const int count = min(pieces, (n + piece - 1) / piece);
  float2* mine = reinterpret_cast<float2*>(scratch) + (size_t)s * pieces * width + c;
  constexpr int kAhead = 8;      // pieces asked for at a time
  for (int p0 = 0; p0 < count; p0 += kAhead) {
    float2 ab[kAhead];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) ab[u] = p0 + u < count ? mine[(size_t)(p0 + u) * width] : make_float2(1.f, 0.f);
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      if (p0 + u < count) mine[(size_t)(p0 + u) * width].y = S;
      S = fmaf(ab[u].x, S, ab[u].y);
    }
  }
}

inline size_t scratch_floats(int n_seqs, int pieces, int width) { return (size_t)n_seqs * pieces * width * 2; }

// pieces 1: one walk; more (with scratch_floats of scratch): pieces of `piece` tokens side by side.
template <typename Rule, typename TOUT>
cudaError_t launch(const Rule& rule, float* state, TOUT* out, const int* seq_slot, const int* seq_start, const int* cu_new,
                   int n_seqs, int width, int piece, int pieces, float* scratch, cudaStream_t stream) {
  const int tiles = (width + kThreads - 1) / kThreads;
  auto walk = [&](auto kernel, int count) {
    return launch_plain(kernel, dim3(n_seqs, tiles, count), dim3(kThreads), 0, stream, rule, state, out, seq_slot, seq_start, cu_new,
                        width, piece, scratch);
  };
  if (pieces == 1) return walk(channel_scan_kernel<0, Rule, TOUT>, 1);
  cudaError_t e = walk(channel_scan_kernel<1, Rule, TOUT>, pieces);
  if (e == cudaSuccess)
    e = launch_plain(channel_carry_kernel, dim3(n_seqs, tiles), dim3(kThreads), 0, stream, scratch, (const float*)state, seq_slot,
                     seq_start, cu_new, width, piece, pieces);
  return e == cudaSuccess ? walk(channel_scan_kernel<2, Rule, TOUT>, pieces) : e;
}

}  // namespace scan
