// Mixture-of-experts routing, token permutation and finalisation.
//
//   moe_route    : softmax / sigmoid scoring (+ selection bias), group-limited top-k
//                  (n_group / topk_group), renormalisation, routed scaling; emits expert ids,
//                  weights, per-expert counts and each token's slot inside its expert
//   moe_offsets  : padded exclusive scan of the counts (segments start on 128-row tiles, so a
//                  GEMM tile never straddles two experts) + the tile -> expert table the grouped
//                  GEMM walks
//   moe_permute  : gather token rows into expert-major order
//   moe_finalize : out[t] = sum_k w[t,k] * y[row(t,k)]  (+ optional shared-expert output)
//   moe_grouped_simt : the grouped products of the fp32 execution type and of odd sizes
//
// Parity: moe_topk_softmax / moe_topk_sigmoid (xllm/core/kernels/cuda/moe/moe_topk_softmax_kernels.cuh,
// moe_topk_sigmoid_kernels.cuh), moe_compute_index (moe_compute_index.cu:37-153) and moe_combine
// (moe_combine.cu:37-102).  The reference's CUDA path drops n_group / topk_group
// (ops_api.cpp:666-671); here group-limited routing (DeepSeek-V3) is implemented.
// Experts outside [expert_begin, expert_end) are not local to this rank (expert parallelism): their
// (token, k) pairs get row -1 and contribute nothing.
#include "vec_io.cuh"

namespace xllm {

constexpr int kMaxExperts = 512;
constexpr int kMaxTopK = 16;
constexpr int kMoeTile = 128;

struct RouteParams {
  const void* logits;   // [T, E] bf16 or fp32, row stride ld
  int64_t ld;
  const float* bias;    // [E] selection bias (e_score_correction_bias) or null
  int32_t* topk_ids;    // [T, K]
  float* topk_w;        // [T, K]
  int32_t* counts;      // [E] zeroed by the caller (or by moe_offsets of the previous call)
  int32_t* slot;        // [T, K] position of the pair inside its expert's segment
  int T, E, K, n_group, topk_group, scoring, renorm, logits_fp32, expert_begin, expert_end, group_max;
  float scale;
};

// one warp per token; lane l owns experts l, l+32, ...
__global__ void __launch_bounds__(128) moe_route_kernel(RouteParams p) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * 4 + warp;
  pdl_wait();
  if (t >= p.T) return;
  constexpr int PER = kMaxExperts / 32;
  float score[PER], sel[PER];
  const int per = (p.E + 31) / 32;
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + i * 32;
    float v = -INFINITY;
    if (i < per && e < p.E)
      v = p.logits_fp32 ? reinterpret_cast<const float*>(p.logits)[t * p.ld + e]
                        : __bfloat162float(reinterpret_cast<const bf16*>(p.logits)[t * p.ld + e]);
    score[i] = v;
    mx = fmaxf(mx, v);
  }
  if (p.scoring == 0) {  // softmax
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      score[i] = (i < per && lane + i * 32 < p.E) ? expf(score[i] - mx) : 0.f;
      sum += score[i];
    }
    sum = warp_sum(sum);
    const float inv = 1.f / sum;
#pragma unroll
    for (int i = 0; i < PER; ++i) score[i] *= inv;
  } else {  // sigmoid
#pragma unroll
    for (int i = 0; i < PER; ++i) score[i] = (i < per && lane + i * 32 < p.E) ? 1.f / (1.f + expf(-score[i])) : 0.f;
  }
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + i * 32;
    sel[i] = (i < per && e < p.E) ? score[i] + (p.bias ? p.bias[e] : 0.f) : -INFINITY;
  }
  // group-limited routing: keep the topk_group groups with the largest score: the sum of a group's two best (with a
  // bias) or its best (without one, or as the caller asks)
  if (p.n_group > 1 && p.topk_group < p.n_group) {
    const int gsz = p.E / p.n_group;
    // group score for every group, computed redundantly by all lanes through shuffles
    float gscore = -INFINITY;  // lane g (< n_group) holds group g's score
    for (int g = 0; g < p.n_group; ++g) {
      float m1 = -INFINITY, m2 = -INFINITY;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int e = lane + i * 32;
        if (i < per && e < p.E && e / gsz == g) {
          const float v = sel[i];
          if (v > m1) { m2 = m1; m1 = v; } else if (v > m2) m2 = v;
        }
      }
      // merge top-2 across lanes
      for (int o = 16; o > 0; o >>= 1) {
        const float o1 = __shfl_xor_sync(0xffffffffu, m1, o), o2 = __shfl_xor_sync(0xffffffffu, m2, o);
        const float a = fmaxf(m1, o1);
        const float b = fmaxf(fminf(m1, o1), fmaxf(m2, o2));
        m1 = a; m2 = b;
      }
      const float gs = p.bias && !p.group_max ? m1 + (m2 > -INFINITY ? m2 : 0.f) : m1;
      if (lane == g) gscore = gs;
    }
    // rank of each group = number of groups with a strictly better score (ties: lower index wins)
    bool keep_group = false;
    {
      int better = 0;
      for (int g = 0; g < p.n_group; ++g) {
        const float og = __shfl_sync(0xffffffffu, gscore, g);
        if (lane < p.n_group && (og > gscore || (og == gscore && g < lane))) ++better;
      }
      keep_group = lane < p.n_group && better < p.topk_group;
    }
    const unsigned keep_mask = __ballot_sync(0xffffffffu, keep_group);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = lane + i * 32;
      if (i < per && e < p.E && !((keep_mask >> (e / gsz)) & 1u)) sel[i] = -INFINITY;
    }
  }
  // iterative top-k by warp arg-max over the selection scores
  float wsum = 0.f;
  float my_w[kMaxTopK];
  int my_id[kMaxTopK];
  for (int k = 0; k < p.K; ++k) {
    float bv = -INFINITY;
    int be = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = lane + i * 32;
      if (i < per && e < p.E && (sel[i] > bv || (sel[i] == bv && e < be))) { bv = sel[i]; be = e; }
    }
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
    }
    // the owner lane supplies the un-biased score as the weight and retires the expert
    float w = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      if (lane + i * 32 == be) { w = score[i]; sel[i] = -INFINITY; }
    }
    w = __shfl_sync(0xffffffffu, w, be & 31);
    my_w[k] = w;
    my_id[k] = be;
    wsum += w;
  }
  const float norm = (p.renorm && wsum > 0.f) ? 1.f / wsum : 1.f;
  if (lane < p.K) {
    // lane k writes pair k
    float w = 0.f;
    int e = 0;
#pragma unroll
    for (int k = 0; k < kMaxTopK; ++k)
      if (k == lane && k < p.K) { w = my_w[k]; e = my_id[k]; }
    p.topk_ids[(int64_t)t * p.K + lane] = e;
    p.topk_w[(int64_t)t * p.K + lane] = w * norm * p.scale;
    int s = -1;
    if (e >= p.expert_begin && e < p.expert_end) s = atomicAdd(&p.counts[e], 1);
    p.slot[(int64_t)t * p.K + lane] = s;
  }
}

// offsets[e] = first row of expert e in the permuted buffer (multiple of 128); tile_expert[i] =
// expert of row tile i (or -1); counts are cleared for the next call; meta[0] = rows used.
__global__ void moe_offsets_kernel(int32_t* counts, int32_t* offsets, int32_t* tile_expert, int32_t* meta, int E,
                                   int max_tiles, int expert_begin) {
  __shared__ int s_off[kMaxExperts + 1];
  if (threadIdx.x == 0) {
    int acc = 0;
    for (int e = 0; e < E; ++e) {
      s_off[e] = acc;
      acc += (counts[e] + kMoeTile - 1) / kMoeTile * kMoeTile;
    }
    s_off[E] = acc;
    meta[0] = acc;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    offsets[e] = s_off[e];
    const int t0 = s_off[e] / kMoeTile, t1 = s_off[e + 1] / kMoeTile;
    for (int i = t0; i < t1 && i < max_tiles; ++i) tile_expert[i] = e - expert_begin;  // index into the local weights
  }
  for (int i = s_off[E] / kMoeTile + threadIdx.x; i < max_tiles; i += blockDim.x) tile_expert[i] = -1;
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) counts[e] = 0;
}

// xp[row(t,k), :] = x[t, :]; rows[t,k] = offsets[e] + slot (or -1 for non-local experts); a row is n_vec vectors of V
template <typename V>
__global__ void __launch_bounds__(256)
moe_permute_kernel(V* __restrict__ xp, int32_t* __restrict__ rows, const V* __restrict__ x, const int32_t* __restrict__ topk_ids,
                   const int32_t* __restrict__ slot, const int32_t* __restrict__ offsets, int T, int K, int n_vec) {
  const int pair = blockIdx.x;
  const int t = pair / K;
  const int s = slot[pair];
  int row = -1;
  if (s >= 0) row = offsets[topk_ids[pair]] + s;
  if (threadIdx.x == 0) rows[pair] = row;
  if (row < 0) return;
  const V* src = x + (int64_t)t * n_vec;
  V* dst = xp + (int64_t)row * n_vec;
  for (int v = threadIdx.x; v < n_vec; v += blockDim.x) dst[v] = src[v];
}

template <typename T_, int V>
__global__ void __launch_bounds__(256)
moe_finalize_kernel(T_* __restrict__ out, const T_* __restrict__ y, int64_t y_ld, const int32_t* __restrict__ rows,
                    const float* __restrict__ w, const T_* __restrict__ shared_out, int T, int K, int H) {
  const int t = blockIdx.x;
  for (int v = threadIdx.x; v < H / V; v += blockDim.x) {
    float acc[V];
    if (shared_out) load_f32<V>(shared_out + (int64_t)t * H + v * V, acc);
    else {
#pragma unroll
      for (int j = 0; j < V; ++j) acc[j] = 0.f;
    }
    for (int k = 0; k < K; ++k) {
      const int row = rows[t * K + k];
      if (row < 0) continue;
      const float wk = w[t * K + k];
      float f[V];
      load_f32<V>(y + (int64_t)row * y_ld + v * V, f);
#pragma unroll
      for (int j = 0; j < V; ++j) acc[j] += wk * f[j];
    }
    store_f32<V>(out + (int64_t)t * H + v * V, acc);
  }
}

// The grouped product without tensor cores, any sizes, fp32 or bf16 operands, fp32 sums: for the fp32 execution type and
// for sizes the tcgen05 kernel does not take.  64 x 64 outputs per CTA, a thread owns 4 x 4; no tile straddles experts.
template <typename T_>
__global__ void __launch_bounds__(256)
moe_grouped_simt_kernel(const T_* __restrict__ a, const T_* __restrict__ w, T_* __restrict__ c, const int32_t* __restrict__ tile_expert,
                        int N, int K, int64_t lda, int64_t ldc) {
  constexpr int BK = 16;
  __shared__ float as[BK][65], ws[BK][65];
  const int m0 = blockIdx.x * 64, n0 = blockIdx.y * 64;
  const int e = tile_expert[m0 / kMoeTile];
  if (e < 0) return;
  const T_* we = w + (int64_t)e * N * K;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
    for (int i = threadIdx.x; i < 64 * BK; i += 256) {
      const int r = i / BK, k = i - r * BK;
      as[k][r] = k0 + k < K ? to_f32(a[(int64_t)(m0 + r) * lda + k0 + k]) : 0.f;
      ws[k][r] = (k0 + k < K && n0 + r < N) ? to_f32(we[(int64_t)(n0 + r) * K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { x[i] = as[k][ty + 16 * i]; y[i] = ws[k][tx + 16 * i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n < N) c[(int64_t)(m0 + ty + 16 * i) * ldc + n] = from_f32<T_>(acc[i][j]);
    }
}

}  // namespace xllm

// scoring: 0 softmax, 1 sigmoid; + 2: groups are ranked by their best score even with a bias.  counts must be zero on entry (moe_offsets re-zeroes it).
XLLM_API int xllm_moe_route_ld(const void* logits, int64_t ld, int logits_fp32, const void* bias, void* topk_ids, void* topk_w,
                               void* counts, void* slot, int T, int E, int K, int n_group, int topk_group, int scoring,
                               int renorm, float scale, int expert_begin, int expert_end, void* stream) {
  using namespace xllm;
  if (T == 0) return 0;
  if (E > kMaxExperts || K > kMaxTopK || K > 32 || n_group > 32 || (n_group > 1 && E % n_group != 0))
    return (int)cudaErrorInvalidValue;
  RouteParams p;
  p.logits = logits; p.ld = ld; p.bias = (const float*)bias; p.topk_ids = (int32_t*)topk_ids; p.topk_w = (float*)topk_w;
  p.counts = (int32_t*)counts; p.slot = (int32_t*)slot; p.T = T; p.E = E; p.K = K; p.n_group = n_group;
  p.topk_group = topk_group; p.scoring = scoring & 1; p.group_max = scoring >> 1; p.renorm = renorm; p.logits_fp32 = logits_fp32;
  p.expert_begin = expert_begin; p.expert_end = expert_end; p.scale = scale;
  moe_route_kernel<<<(T + 3) / 4, 128, 0, (cudaStream_t)stream>>>(p);
  return XLLM_LAUNCH_CHECK();
}

// the same with dense logits
XLLM_API int xllm_moe_route(const void* logits, int logits_fp32, const void* bias, void* topk_ids, void* topk_w,
                            void* counts, void* slot, int T, int E, int K, int n_group, int topk_group, int scoring,
                            int renorm, float scale, int expert_begin, int expert_end, void* stream) {
  return xllm_moe_route_ld(logits, E, logits_fp32, bias, topk_ids, topk_w, counts, slot, T, E, K, n_group, topk_group, scoring,
                           renorm, scale, expert_begin, expert_end, stream);
}

XLLM_API int xllm_moe_offsets(void* counts, void* offsets, void* tile_expert, void* meta, int E, int max_tiles,
                              int expert_begin, void* stream) {
  using namespace xllm;
  moe_offsets_kernel<<<1, 256, 0, (cudaStream_t)stream>>>((int32_t*)counts, (int32_t*)offsets, (int32_t*)tile_expert,
                                                         (int32_t*)meta, E, max_tiles, expert_begin);
  return XLLM_LAUNCH_CHECK();
}

// dtype of the entry points below: 0 bf16, 1 fp32.
XLLM_API int xllm_moe_permute(void* xp, void* rows, const void* x, const void* topk_ids, const void* slot,
                              const void* offsets, int T, int K, int H, int dtype, void* stream) {
  using namespace xllm;
  if (T == 0) return 0;
  const auto run = [&](auto tag, int n_vec) {
    using V = decltype(tag);
    moe_permute_kernel<V><<<T * K, 256, 0, (cudaStream_t)stream>>>((V*)xp, (int32_t*)rows, (const V*)x, (const int32_t*)topk_ids,
                                                                  (const int32_t*)slot, (const int32_t*)offsets, T, K, n_vec);
  };
  const int bytes = H * (dtype == 0 ? 2 : 4);
  if (bytes % 16 == 0 && (((uintptr_t)xp | (uintptr_t)x) & 15) == 0) run(uint4(), bytes / 16);
  else run((unsigned short)0, bytes / 2);
  return XLLM_LAUNCH_CHECK();
}

// y: rows of y_ld elements, of which the first H count
XLLM_API int xllm_moe_finalize(void* out, const void* y, int64_t y_ld, const void* rows, const void* w, const void* shared_out,
                               int T, int K, int H, int dtype, void* stream) {
  using namespace xllm;
  if (T == 0) return 0;
  const bool v8 = H % 8 == 0 && y_ld % 8 == 0 && (((uintptr_t)out | (uintptr_t)y | (uintptr_t)shared_out) & 15) == 0;
  const auto run = [&](auto tag, auto kernel) {
    using E = decltype(tag);
    kernel<<<T, 256, 0, (cudaStream_t)stream>>>((E*)out, (const E*)y, y_ld, (const int32_t*)rows, (const float*)w,
                                                (const E*)shared_out, T, K, H);
  };
  if (dtype == 0) {
    if (v8) run(bf16(), moe_finalize_kernel<bf16, 8>);
    else run(bf16(), moe_finalize_kernel<bf16, 1>);
  } else {
    if (v8) run(float(), moe_finalize_kernel<float, 8>);
    else run(float(), moe_finalize_kernel<float, 1>);
  }
  return XLLM_LAUNCH_CHECK();
}

// C[M, N] = A[M, K] W[expert of the 128-row tile]^T, w [experts, N, K]; M a multiple of 128.  Rows of unused tiles are left.
XLLM_API int xllm_moe_grouped_simt(const void* a, const void* w, void* c, const void* tile_expert, int M, int N, int K,
                                   int64_t lda, int64_t ldc, int dtype, void* stream) {
  using namespace xllm;
  if (M == 0 || N == 0) return 0;
  if (M % kMoeTile || K <= 0) return (int)cudaErrorInvalidValue;
  const dim3 grid(M / 64, (N + 63) / 64);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == 0)
    moe_grouped_simt_kernel<bf16><<<grid, 256, 0, s>>>((const bf16*)a, (const bf16*)w, (bf16*)c, (const int32_t*)tile_expert, N, K, lda, ldc);
  else
    moe_grouped_simt_kernel<float><<<grid, 256, 0, s>>>((const float*)a, (const float*)w, (float*)c, (const int32_t*)tile_expert, N, K, lda, ldc);
  return XLLM_LAUNCH_CHECK();
}
