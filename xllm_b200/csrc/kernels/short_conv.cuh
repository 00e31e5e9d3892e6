// Short causal convolution over time per channel, followed by silu, over projection rows as the GEMM left them.
//
// A sequence keeps its last inputs in a ring of `taps` rows per state slot, row (position mod taps): the token at
// position p reads positions p - 1 .. p - taps + 1 and may store its own row at any time, since no token of the same
// step that reads the ring needs that row from it.  Positions before 0 are zeros, so a fresh sequence needs no reset.
#pragma once
#include "vec_io.cuh"

namespace xllm {

__device__ __forceinline__ float sigmoid_exact(float z) { return 1.f / (1.f + expf(-z)); }

// V neighbouring channels of one token.  x: the channels' place in the token's projection row (row stride ld); `back`:
// how many rows before it belong to the same sequence in this batch; ring, w: the channels' place in row 0 of the slot's
// ring and of the weights [taps, C] (the last row belongs to the current token).
template <typename T, int V>
__device__ __forceinline__ void conv_silu(const T* x, int64_t ld, int back, int pos, const T* ring, int64_t C, const T* w,
                                          int taps, float* y) {
#pragma unroll
  for (int j = 0; j < V; ++j) y[j] = 0.f;
  for (int d = 0; d < taps && d <= pos; ++d) {
    float v[V], f[V];
    if (d <= back) load_f32<V>(x - d * ld, v);
    else load_f32<V>(ring + (int64_t)((pos - d) % taps) * C, v);
    load_f32<V>(w + (int64_t)(taps - 1 - d) * C, f);
#pragma unroll
    for (int j = 0; j < V; ++j) y[j] += v[j] * f[j];
  }
#pragma unroll
  for (int j = 0; j < V; ++j) y[j] = silu_as<T>(y[j]);
}

// the sequence b with cu_q[b] <= row < cu_q[b + 1], or -1
__device__ __forceinline__ int seq_of_row(const int32_t* cu_q, int n_seqs, int row) {
  if (row < cu_q[0] || row >= cu_q[n_seqs]) return -1;
  int lo = 0, hi = n_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi) >> 1;
    if (cu_q[mid + 1] > row) hi = mid;
    else lo = mid + 1;
  }
  return lo;
}

}  // namespace xllm
