// Paged causal GQA attention for the cases the tensor-core kernels do not take: fp32 caches and head sizes
// beyond 256 (with a window the first `keep` positions may stay visible; scores may be bounded by a soft cap).  Decode rows and prompt chunks alike: row r of sequence b sees the cache positions
// [0, kv_len_b - (rows of b after r)).  One CTA per (query row, head); each of its four warps walks every
// fourth key with its lanes over the head dimension, keeps a running softmax, and the four are merged at the end.
#include "vec_io.cuh"

namespace xllm {

template <typename T>
struct GenericAttnParams {
  const T* q;              // [T, nq, d]
  T* out;
  const T* k_cache;        // [n_blocks, nkv, page, d]
  const T* v_cache;
  const int32_t* block_table;
  const int32_t* cu_q;     // [n_seqs + 1]
  const int32_t* kv_lens;
  int64_t q_ld, o_ld;
  int bt_stride, n_seqs, nq, nkv, d, page, row0, window, keep;
  float scale, softcap;
};

template <typename T, int NPL>
__global__ void __launch_bounds__(128) attn_generic_kernel(GenericAttnParams<T> p) {
  __shared__ float sm_m[4], sm_l[4];
  __shared__ float sm_o[4][NPL * 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = p.row0 + blockIdx.x, h = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  if (row < p.cu_q[0] || row >= p.cu_q[p.n_seqs]) return;
  int lo = 0, hi = p.n_seqs - 1;                    // the sequence b with cu_q[b] <= row < cu_q[b + 1]
  while (lo < hi) {
    const int mid = (lo + hi) >> 1;
    if (p.cu_q[mid + 1] > row) hi = mid; else lo = mid + 1;
  }
  const int b = lo;
  const int len = p.kv_lens[b] - (p.cu_q[b + 1] - 1 - row);
  const int first = p.window > 0 ? max(0, len - p.window) : 0;
  const int kept = min(p.keep, first), keys = kept + len - first;       // the walk: 0 .. kept - 1, then first .. len - 1
  const int g = h / (p.nq / p.nkv);
  const T* qr = p.q + (int64_t)row * p.q_ld + (int64_t)h * p.d;
  const int32_t* bt = p.block_table + (int64_t)b * p.bt_stride;
  float q[NPL], o[NPL];
#pragma unroll
  for (int i = 0; i < NPL; ++i) {
    const int c = lane + 32 * i;
    q[i] = c < p.d ? to_f32(qr[c]) * p.scale : 0.f;
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int n = warp; n < keys; n += 4) {
    const int j = n < kept ? n : n - kept + first;
    const int pg = j / p.page;
    const int64_t base = (((int64_t)bt[pg] * p.nkv + g) * p.page + (j - pg * p.page)) * p.d;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      const int c = lane + 32 * i;
      if (c < p.d) s += q[i] * to_f32(p.k_cache[base + c]);
    }
    s = warp_sum(s);
    if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    const float mn = fmaxf(m, s);
    const float keep = expf(m - mn), w = expf(s - mn);
    m = mn;
    l = l * keep + w;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      const int c = lane + 32 * i;
      o[i] = o[i] * keep + (c < p.d ? w * to_f32(p.v_cache[base + c]) : 0.f);
    }
  }
  if (lane == 0) { sm_m[warp] = m; sm_l[warp] = l; }
#pragma unroll
  for (int i = 0; i < NPL; ++i) sm_o[warp][lane + 32 * i] = o[i];
  __syncthreads();
  float M = -INFINITY;
  for (int w = 0; w < 4; ++w) M = fmaxf(M, sm_m[w]);
  float L = 0.f, wt[4];
  for (int w = 0; w < 4; ++w) {
    wt[w] = M > -INFINITY ? expf(sm_m[w] - M) : 0.f;
    L += sm_l[w] * wt[w];
  }
  T* orow = p.out + (int64_t)row * p.o_ld + (int64_t)h * p.d;
  for (int c = threadIdx.x; c < p.d; c += 128) {
    float a = 0.f;
    for (int w = 0; w < 4; ++w) a += sm_o[w][c] * wt[w];
    orow[c] = from_f32<T>(L > 0.f ? a / L : 0.f);
  }
}

}  // namespace xllm

// Rows [row0, row0 + rows) of q / out; dtype: 0 bf16, 1 fp32; d <= 1024.
XLLM_API int xllm_paged_attn_generic(void* out, int64_t o_ld, const void* q, int64_t q_ld, const void* k_cache,
                                     const void* v_cache, const void* block_table, int bt_stride, const void* cu_q,
                                     const void* kv_lens, int n_seqs, int row0, int rows, int nq, int nkv, int d, int page,
                                     float scale, int window, int keep, float softcap, int dtype, void* stream) {
  using namespace xllm;
  if (rows == 0 || n_seqs == 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv != 0 || d <= 0 || d > 1024 || page <= 0 || keep < 0) return (int)cudaErrorInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    GenericAttnParams<T> p;
    p.q = (const T*)q; p.out = (T*)out; p.k_cache = (const T*)k_cache; p.v_cache = (const T*)v_cache;
    p.block_table = (const int32_t*)block_table; p.cu_q = (const int32_t*)cu_q; p.kv_lens = (const int32_t*)kv_lens;
    p.q_ld = q_ld; p.o_ld = o_ld; p.bt_stride = bt_stride; p.n_seqs = n_seqs; p.nq = nq; p.nkv = nkv; p.d = d;
    p.page = page; p.row0 = row0; p.window = window; p.scale = scale;
    p.keep = window > 0 ? keep : 0; p.softcap = softcap;
    const dim3 grid(rows, nq);
    if (d <= 64) launch_pdl(attn_generic_kernel<T, 2>, grid, dim3(128), 0, s, p);
    else if (d <= 128) launch_pdl(attn_generic_kernel<T, 4>, grid, dim3(128), 0, s, p);
    else if (d <= 256) launch_pdl(attn_generic_kernel<T, 8>, grid, dim3(128), 0, s, p);
    else if (d <= 512) launch_pdl(attn_generic_kernel<T, 16>, grid, dim3(128), 0, s, p);
    else launch_pdl(attn_generic_kernel<T, 32>, grid, dim3(128), 0, s, p);
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return XLLM_LAUNCH_CHECK();
}
