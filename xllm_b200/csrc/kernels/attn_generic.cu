// Paged causal GQA attention for the cases the tensor-core kernels do not take: fp32 caches and head sizes
// beyond 256 (with a window the first `keep` positions may stay visible; scores may be bounded by a soft cap;
// a sink per head may join the denominator).  Decode rows and prompt chunks alike: row r of sequence b sees the cache positions
// [0, kv_len_b - (rows of b after r)).  One CTA per (query row, head); each of its four warps walks every
// fourth key with its lanes over the head dimension, keeps a running softmax, and the four are merged at the end.
//
// Also here, for any size and fp32: attention whose heads' softmax weights are mixed by a matrix before they meet the values
// ("talking heads"), in three launches over a table of weights [rows, heads, keys] (attn_talk.cu has the tensor-core form).
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
  const float* sink;       // [nq] or null
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
  if (p.sink != nullptr && warp == 0) {             // a key with this score and no value
    m = p.sink[h];
    l = 1.f;
  }
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

template <typename T>
struct TalkParams {
  const T* q;              // [T, nq, d_pad]
  T* out;                  // [T, nq, dv]
  const T *k_cache, *v_cache;   // [n_blocks, nkv, page, d_pad]
  const T* talk;           // [nq, nq]
  float* w;                // [rows, nq, ld]
  const int32_t *block_table, *cu_q, *kv_lens;
  int64_t ld;
  int bt_stride, n_seqs, nq, nkv, d, dv, d_pad, page, row0;
  float scale, softcap;
};

// sequence and visible keys of a row; false: the row belongs to no sequence
template <typename T>
__device__ __forceinline__ bool talk_row(const TalkParams<T>& p, int row, int& b, int& len) {
  if (row < p.cu_q[0] || row >= p.cu_q[p.n_seqs]) return false;
  int lo = 0, hi = p.n_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi) >> 1;
    if (p.cu_q[mid + 1] > row) hi = mid; else lo = mid + 1;
  }
  b = lo;
  len = p.kv_lens[b] - (p.cu_q[b + 1] - 1 - row);
  return len > 0;
}

constexpr int kTalkKeys = 64;

// grid (rows, key tiles): capped scores of all heads; a warp takes every fourth key of the tile, its lanes the head dimension
template <typename T>
__global__ void __launch_bounds__(128) talk_scores_kernel(TalkParams<T> p) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = p.row0 + blockIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  int b, len;
  if (!talk_row(p, row, b, len)) return;
  const int j0 = blockIdx.y * kTalkKeys, group = p.nq / p.nkv;
  float* w = p.w + (int64_t)blockIdx.x * p.nq * p.ld;
  for (int j = j0 + warp; j < min(len, j0 + kTalkKeys); j += 4) {
    const int pg = j / p.page;
    const int64_t blk = p.block_table[(int64_t)b * p.bt_stride + pg];
    for (int h = 0; h < p.nq; ++h) {
      const T* k = p.k_cache + ((blk * p.nkv + h / group) * p.page + (j - pg * p.page)) * p.d_pad;
      const T* q = p.q + ((int64_t)row * p.nq + h) * p.d_pad;
      float s = 0.f;
      for (int c = lane; c < p.d; c += 32) s += to_f32(q[c]) * to_f32(k[c]);
      s = warp_sum(s) * p.scale;
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      if (lane == 0) w[h * p.ld + j] = s;
    }
  }
}

// one CTA per row: softmax of every head, then the mixture, in place; shared memory 2 nq + nq * kTalkKeys floats
template <typename T>
__global__ void __launch_bounds__(256) talk_mix_kernel(TalkParams<T> p) {
  extern __shared__ float sm[];
  float *top = sm, *inv = sm + p.nq, *tile = inv + p.nq;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = p.row0 + blockIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  int b, len;
  if (!talk_row(p, row, b, len)) return;
  float* w = p.w + (int64_t)blockIdx.x * p.nq * p.ld;
  for (int h = warp; h < p.nq; h += 8) {
    float m = -INFINITY, l = 0.f;
    for (int j = lane; j < len; j += 32) m = fmaxf(m, w[h * p.ld + j]);
    m = warp_max(m);
    for (int j = lane; j < len; j += 32) l += expf(w[h * p.ld + j] - m);
    l = warp_sum(l);
    if (lane == 0) {
      top[h] = m;
      inv[h] = 1.f / l;
    }
  }
  for (int j0 = 0; j0 < len; j0 += kTalkKeys) {
    __syncthreads();
    const int n = min(kTalkKeys, len - j0);
    for (int i = threadIdx.x; i < p.nq * kTalkKeys; i += 256) {
      const int h = i / kTalkKeys, j = i - h * kTalkKeys;
      if (j < n) tile[i] = expf(w[h * p.ld + j0 + j] - top[h]) * inv[h];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.nq * kTalkKeys; i += 256) {
      const int h = i / kTalkKeys, j = i - h * kTalkKeys;
      if (j >= n) continue;
      float a = 0.f;
      for (int g = 0; g < p.nq; ++g) a += to_f32(p.talk[h * p.nq + g]) * tile[g * kTalkKeys + j];
      w[h * p.ld + j0 + j] = a;
    }
  }
}

// grid (rows, heads): mixed weights times values; four warps walk every fourth key
template <typename T, int NPL>
__global__ void __launch_bounds__(128) talk_values_kernel(TalkParams<T> p) {
  __shared__ float sm_o[4][NPL * 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = p.row0 + blockIdx.x, h = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  int b, len;
  if (!talk_row(p, row, b, len)) return;
  const float* w = p.w + ((int64_t)blockIdx.x * p.nq + h) * p.ld;
  const int g = h / (p.nq / p.nkv);
  float o[NPL];
#pragma unroll
  for (int i = 0; i < NPL; ++i) o[i] = 0.f;
  for (int j = warp; j < len; j += 4) {
    const int pg = j / p.page;
    const T* v = p.v_cache + (((int64_t)p.block_table[(int64_t)b * p.bt_stride + pg] * p.nkv + g) * p.page + (j - pg * p.page)) * p.d_pad;
    const float x = w[j];
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      const int c = lane + 32 * i;
      if (c < p.dv) o[i] += x * to_f32(v[c]);
    }
  }
#pragma unroll
  for (int i = 0; i < NPL; ++i) sm_o[warp][lane + 32 * i] = o[i];
  __syncthreads();
  for (int c = threadIdx.x; c < p.dv; c += 128)
    p.out[((int64_t)row * p.nq + h) * p.dv + c] = from_f32<T>(sm_o[0][c] + sm_o[1][c] + sm_o[2][c] + sm_o[3][c]);
}

}  // namespace xllm

// Rows [row0, row0 + rows) of q / out; dtype: 0 bf16, 1 fp32; d <= 1024.
XLLM_API int xllm_paged_attn_generic(void* out, int64_t o_ld, const void* q, int64_t q_ld, const void* k_cache,
                                     const void* v_cache, const void* block_table, int bt_stride, const void* cu_q,
                                     const void* kv_lens, int n_seqs, int row0, int rows, int nq, int nkv, int d, int page,
                                     float scale, int window, int keep, float softcap, const void* sink, int dtype, void* stream) {
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
    p.keep = window > 0 ? keep : 0; p.softcap = softcap; p.sink = (const float*)sink;
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

// Rows [row0, row0 + rows) of q [T, nq, d_pad] / out [T, nq, dv]: causal attention with capped scores (softcap > 0) whose softmax
// weights are mixed, weight_h <- sum_g talk[h, g] weight_g, before head h's values.  w: rows * nq * ld floats, ld >= the longest
// sequence.  dtype: 0 bf16, 1 fp32; dv <= 1024.
XLLM_API int xllm_talk_attn_generic(void* out, const void* q, const void* k_cache, const void* v_cache, const void* talk, void* w,
                                    int64_t ld, const void* block_table, int bt_stride, const void* cu_q, const void* kv_lens,
                                    int n_seqs, int row0, int rows, int nq, int nkv, int d, int dv, int d_pad, int page, float scale,
                                    float softcap, int dtype, void* stream) {
  using namespace xllm;
  if (rows == 0 || n_seqs == 0) return 0;
  const size_t smem = (size_t)nq * (2 + kTalkKeys) * 4;
  if (nq <= 0 || nkv <= 0 || nq % nkv != 0 || d <= 0 || dv <= 0 || dv > 1024 || d_pad < d || d_pad < dv || page <= 0 || ld <= 0 ||
      w == nullptr || talk == nullptr || smem > 200 * 1024)
    return (int)cudaErrorInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  const auto run = [&](auto tag) -> int {
    using T = decltype(tag);
    TalkParams<T> p{(const T*)q, (T*)out, (const T*)k_cache, (const T*)v_cache, (const T*)talk, (float*)w, (const int32_t*)block_table,
                    (const int32_t*)cu_q, (const int32_t*)kv_lens, ld, bt_stride, n_seqs, nq, nkv, d, dv, d_pad, page, row0, scale,
                    softcap};
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(talk_mix_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    launch_pdl(talk_scores_kernel<T>, dim3(rows, (unsigned)((ld + kTalkKeys - 1) / kTalkKeys)), dim3(128), 0, s, p);
    launch_pdl(talk_mix_kernel<T>, dim3(rows), dim3(256), smem, s, p);
    const dim3 grid(rows, nq);
    if (dv <= 64) launch_pdl(talk_values_kernel<T, 2>, grid, dim3(128), 0, s, p);
    else if (dv <= 128) launch_pdl(talk_values_kernel<T, 4>, grid, dim3(128), 0, s, p);
    else if (dv <= 256) launch_pdl(talk_values_kernel<T, 8>, grid, dim3(128), 0, s, p);
    else launch_pdl(talk_values_kernel<T, 32>, grid, dim3(128), 0, s, p);
    return XLLM_LAUNCH_CHECK();
  };
  return dtype == 0 ? run(bf16()) : run(float());
}
