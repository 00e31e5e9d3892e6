// Paged causal attention whose heads' softmax weights are mixed by a matrix before they meet the values ("talking heads" behind the
// softmax), scores softly capped: bf16, cached heads of 128 (smaller ones zero-padded).
//
//   p_g(i, j) = softmax_j(cap(scale q_g . k_c(g)(j)));   w_h(i, j) = sum_g T[h, g] p_g(i, j);   out_h(i) = sum_j w_h(i, j) v_c(h)(j)
//
// A mixed weight needs every head's normalised weight of its pair, so the softmax's sums come first and the weights exist as a
// table for a while.  Nothing below is rounded to bf16 but operands of products: the weights enter the mixture as two bf16 terms
// (T is bf16 as stored), and the mixture is rounded as the operand of its product with V.
//
// Decoding, three launches:
//   talk_scores_tc_kernel   capped scores of a split of the context to the table, with the split's maximum and sum per head
//   talk_decode_kernel      a block of 64 keys at a time: weights of all heads, mixture, product with the values of eight units
//                           (a unit: up to 16 heads of one key/value head); two splits or more leave partial sums
//   talk_merge_kernel       adds them
// Prompts: the log-sum-exp of every row (xllm_prefill_lse_tc), then
//   talk_weights_kernel     mixed weights of 16 rows and a range of keys to the table
// and its product with the values (xllm_talk_values_tc).
//
// The mixture of 16 rows: a warp owns up to four heads of one key/value head, whose queries stay in registers, and makes the
// transposed scores [16 keys x 8 rows] of each (mma.sync m16n8k16, keys as M), so that it has the weights of four heads for its
// pairs and stores them as one 16-byte chunk of a pair's line: four leading terms, four remainders.  The lines of all units are the
// B operand of the mixture (pairs as N, chunks as K), T repeated for leading terms and remainders the A operand, and what comes
// out is four neighbouring keys per thread.  A step's mixture is computed beside the next step's scores.
#include "attn_common.cuh"
#include <atomic>

namespace xllm {
namespace talk {

constexpr int D = 128, CH = D / 8;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float score(float s, const SoftCap& cap, float scale_log2) {
  return cap.out > 0.f ? soft_cap(s, cap) : s * scale_log2;
}

// ------------------------------------------------------------------------------------------------ decoding
struct DecodeParams {
  const bf16* q;              // [B, nq, 128]
  const bf16 *k_cache, *v_cache;   // [n_blocks, nkv, page, 128]
  const bf16* talk;           // [nq, nq]
  bf16* out;                  // [B, nq, dv]
  float* s;                   // [B, nq, ld] scores, log2 domain
  float2* stat;               // [B, nq, splits] maximum and sum of every split of the scores
  float* part;                // [B, nq, vsplits, 128]
  const int32_t *block_table, *seq_lens;
  int64_t ld;
  int bt_stride, nq, nkv, group, page, splits, vsplits, dv;
  SoftCap cap;
  float scale_log2;
};

constexpr int kScoreStages = 4, kTileBytes = 16 * D * 2;

// grid (kv heads * tiles of 16 heads, batch, splits), 4 warps; each walks every fourth tile of 16 keys through a ring of its own
__global__ void __launch_bounds__(128) talk_scores_tc_kernel(DecodeParams p) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float sm_m[4][16], sm_l[4][16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qtiles = (p.group + 15) >> 4, kvh = blockIdx.x / qtiles, qt = blockIdx.x - kvh * qtiles;
  const int b = blockIdx.y, split = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  const int len = p.seq_lens[b];
  const int tiles = (len + 15) >> 4, tps = (tiles + p.splits - 1) / p.splits;
  const int t0 = split * tps, my_n = (min(t0 + tps, tiles) - t0 - warp + 3) >> 2;
  const int rows = min(16, p.group - qt * 16), head0 = kvh * p.group + qt * 16;
  const int r0 = lane >> 2, r1 = r0 + 8;
  uint32_t qa[8][4];
  {
    const bf16* qb = p.q + ((int64_t)b * p.nq + head0) * D;
#pragma unroll
    for (int ks = 0; ks < 8; ++ks) {
      const int col = ks * 16 + (lane & 3) * 2;
      qa[ks][0] = r0 < rows ? *reinterpret_cast<const uint32_t*>(qb + r0 * D + col) : 0u;
      qa[ks][1] = r1 < rows ? *reinterpret_cast<const uint32_t*>(qb + r1 * D + col) : 0u;
      qa[ks][2] = r0 < rows ? *reinterpret_cast<const uint32_t*>(qb + r0 * D + col + 8) : 0u;
      qa[ks][3] = r1 < rows ? *reinterpret_cast<const uint32_t*>(qb + r1 * D + col + 8) : 0u;
    }
  }
  const uint32_t ring = smem_u32(smem) + warp * (kScoreStages * kTileBytes);
  const int32_t* bt = p.block_table + (int64_t)b * p.bt_stride;
  const auto load = [&](int i) {
    if (i < my_n) {
      const int tok0 = (t0 + warp + 4 * i) << 4, pg = tok0 / p.page;
      const bf16* kb = p.k_cache + (((int64_t)bt[pg] * p.nkv + kvh) * p.page + tok0 - pg * p.page) * D;
      const uint32_t dst = ring + (i % kScoreStages) * kTileBytes;
#pragma unroll
      for (int j = 0; j < 16 * CH / 32; ++j) {
        const int id = lane + j * 32, r = id / CH, c = id - r * CH;
        const bool in = tok0 + r < len;
        cp_async16(dst + swz<CH>(r, c), kb + (in ? r * D + c * 8 : 0), in);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < kScoreStages - 1; ++i) load(i);
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  float *w0 = p.s + ((int64_t)b * p.nq + head0 + r0) * p.ld, *w1 = w0 + 8 * p.ld;
  for (int i = 0; i < my_n; ++i) {
    cp_async_wait<kScoreStages - 2>();
    __syncwarp();
    load(i + kScoreStages - 1);
    const uint32_t ka = ring + (i % kScoreStages) * kTileBytes;
    const int tok0 = (t0 + warp + 4 * i) << 4;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const int row = (lane & 7) + ((lane >> 4) << 3), cb = (lane >> 3) & 1;
#pragma unroll
    for (int ks = 0; ks < 8; ++ks) {
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4(b0, b1, b2, b3, ka + swz<CH>(row, ks * 2 + cb));
      mma_bf16_16816(s[0], qa[ks], b0, b1);
      mma_bf16_16816(s[1], qa[ks], b2, b3);
    }
    float x0 = m0, x1 = m1;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int tok = tok0 + nt * 8 + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s[nt][j] = tok + (j & 1) < len ? score(s[nt][j], p.cap, p.scale_log2) : -INFINITY;
        if (j < 2) x0 = fmaxf(x0, s[nt][j]); else x1 = fmaxf(x1, s[nt][j]);
      }
      if (r0 < rows) *reinterpret_cast<float2*>(w0 + tok) = make_float2(s[nt][0], s[nt][1]);
      if (r1 < rows) *reinterpret_cast<float2*>(w1 + tok) = make_float2(s[nt][2], s[nt][3]);
    }
    // a lane keeps the sums of its own columns; a reference of 0 while it has seen none
    const float f0 = x0 == -INFINITY ? 0.f : x0, f1 = x1 == -INFINITY ? 0.f : x1;
    l0 = l0 * exp2f(m0 - f0) + exp2f(s[0][0] - f0) + exp2f(s[0][1] - f0) + exp2f(s[1][0] - f0) + exp2f(s[1][1] - f0);
    l1 = l1 * exp2f(m1 - f1) + exp2f(s[0][2] - f1) + exp2f(s[0][3] - f1) + exp2f(s[1][2] - f1) + exp2f(s[1][3] - f1);
    m0 = x0;
    m1 = x1;
  }
  cp_async_wait<0>();
#pragma unroll
  for (int o = 1; o < 4; o <<= 1) {
    const float a0 = __shfl_xor_sync(0xffffffffu, m0, o), a1 = __shfl_xor_sync(0xffffffffu, m1, o);
    const float b0 = __shfl_xor_sync(0xffffffffu, l0, o), b1 = __shfl_xor_sync(0xffffffffu, l1, o);
    const float n0 = fmaxf(m0, a0), n1 = fmaxf(m1, a1), f0 = n0 == -INFINITY ? 0.f : n0, f1 = n1 == -INFINITY ? 0.f : n1;
    l0 = l0 * exp2f(m0 - f0) + b0 * exp2f(a0 - f0);
    l1 = l1 * exp2f(m1 - f1) + b1 * exp2f(a1 - f1);
    m0 = n0;
    m1 = n1;
  }
  if ((lane & 3) == 0) {
    sm_m[warp][r0] = m0; sm_m[warp][r1] = m1;
    sm_l[warp][r0] = l0; sm_l[warp][r1] = l1;
  }
  __syncthreads();
  if ((int)threadIdx.x < rows) {
    const int r = threadIdx.x;
    float m = -INFINITY, l = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, sm_m[w][r]);
#pragma unroll
    for (int w = 0; w < 4; ++w) l += m > -INFINITY ? sm_l[w][r] * exp2f(sm_m[w][r] - m) : 0.f;
    p.stat[((int64_t)b * p.nq + head0 + r) * p.splits + split] = make_float2(m, l);
  }
}

constexpr int kKeys = 64, kValueStages = 3, kMaxHeads = 64;

// 16-byte chunk c of row r in a tile of rows of C chunks (2, 4, 8 or 16): eight rows of one chunk column hit different banks
template <int C>
__device__ __forceinline__ uint32_t slice(int r, int c) {
  constexpr int per = C >= 8 ? 1 : 8 / C;             // rows in 128 bytes
  return (uint32_t)((r * C + (c ^ ((r / per) & (C >= 8 ? 7 : C - 1)))) << 4);
}

// grid (groups of 8 / WPU units, batch, splits), 8 warps.  WPU warps share a unit, each with 128 / WPU columns of the values.
// Dynamic shared memory: value rings, mixture [2][nq + 16][64] bf16, weights [nq][64], T [nq][nq], log-sum-exps [nq].
template <int WPU>
__global__ void __launch_bounds__(256) talk_decode_kernel(DecodeParams p) {
  constexpr int NC = D / WPU, C = NC / 8, VT = 16 * NC * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nq = p.nq;
  const int qtiles = (p.group + 15) >> 4, units = p.nkv * qtiles;
  const int unit = blockIdx.x * (8 / WPU) + warp / WPU, col0 = warp % WPU * NC;
  const bool mine = unit < units;
  const int kvh = mine ? unit / qtiles : 0, qt = unit - kvh * qtiles;
  const int rows = mine ? min(16, p.group - qt * 16) : 0, head0 = kvh * p.group + (mine ? qt * 16 : 0);
  const int b = blockIdx.y, split = blockIdx.z;
  const uint32_t ring = smem_u32(smem) + warp * (kValueStages * VT), wbuf = smem_u32(smem) + 8 * kValueStages * VT;
  const int wrows = nq + 16;
  uint8_t* wptr = smem + 8 * kValueStages * VT;
  float *pt = reinterpret_cast<float*>(wptr + 2 * wrows * kKeys * 2), *tt = pt + nq * kKeys, *lse = tt + nq * nq;
  pdl_wait();
  pdl_launch_dependents();
  const int len = p.seq_lens[b];
  const int blocks = (len + kKeys - 1) / kKeys, bps = (blocks + p.vsplits - 1) / p.vsplits;
  const int b0 = split * bps, nb = max(0, min(b0 + bps, blocks) - b0), nt = nb * (kKeys / 16);
  const int32_t* bt = p.block_table + (int64_t)b * p.bt_stride;
  const auto load = [&](int i) {                      // i-th tile of 16 values
    const int tok0 = b0 * kKeys + i * 16;
    if (mine && i < nt && tok0 < len) {
      const int pg = tok0 / p.page;
      const bf16* vb = p.v_cache + (((int64_t)bt[pg] * p.nkv + kvh) * p.page + tok0 - pg * p.page) * D + col0;
      const uint32_t dst = ring + (i % kValueStages) * VT;
#pragma unroll
      for (int j = 0; j < 16 * C / 32; ++j) {
        const int id = lane + j * 32, r = id / C, c = id - r * C;
        const bool in = tok0 + r < len;
        cp_async16(dst + slice<C>(r, c), vb + (in ? r * D + c * 8 : 0), in);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < kValueStages - 1; ++i) load(i);
  for (int i = threadIdx.x; i < nq * nq; i += 256) tt[i] = __bfloat162float(p.talk[i]);
  for (int i = threadIdx.x; i < 16 * kKeys; i += 256) {          // rows behind the last head: operands of products nobody keeps
    reinterpret_cast<bf16*>(wptr)[nq * kKeys + i] = __float2bfloat16(0.f);
    reinterpret_cast<bf16*>(wptr)[(wrows + nq) * kKeys + i] = __float2bfloat16(0.f);
  }
  for (int h = threadIdx.x; h < nq; h += 256) {
    const float2* st = p.stat + ((int64_t)b * nq + h) * p.splits;
    float m = -INFINITY, l = 0.f;
    for (int s = 0; s < p.splits; ++s) m = fmaxf(m, st[s].x);
    for (int s = 0; s < p.splits; ++s) l += m > -INFINITY ? st[s].y * exp2f(st[s].x - m) : 0.f;
    lse[h] = l > 0.f ? m + log2f(l) : INFINITY;
  }
  float o[NC / 8][4];
#pragma unroll
  for (int i = 0; i < NC / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int key = threadIdx.x & 63, hg = threadIdx.x >> 6;        // heads hg, hg + 4, ...
  const float* srow = p.s + (int64_t)b * nq * p.ld;
  float next[kMaxHeads / 4];
  const auto fetch = [&](int blk) {
    const int j = (b0 + blk) * kKeys + key;
#pragma unroll
    for (int i = 0; i < kMaxHeads / 4; ++i) {
      const int h = hg + 4 * i;
      next[i] = h < nq && blk < nb && j < len ? srow[h * p.ld + j] : -INFINITY;
    }
  };
  fetch(0);
  __syncthreads();
  for (int blk = 0; blk < nb; ++blk) {
#pragma unroll
    for (int i = 0; i < kMaxHeads / 4; ++i) {
      const int h = hg + 4 * i;
      if (h < nq) pt[h * kKeys + key] = exp2f(next[i] - lse[h]);
    }
    fetch(blk + 1);
    __syncthreads();
    const uint32_t wcur = wbuf + (blk & 1) * wrows * kKeys * 2;
    {
      // the heads of a thread: hg, hg + 4, ... in groups of four that share the loads of the weights
      uint8_t* wrow = wptr + (blk & 1) * wrows * kKeys * 2;
      for (int h = hg; h < nq; h += 16) {
        float a[4] = {0.f, 0.f, 0.f, 0.f};
        const int n = min(4, (nq - h + 3) >> 2);
        int g = 0;
        if (nq % 4 == 0) {
#pragma unroll 2
          for (; g < nq; g += 4) {
            float x[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) x[e] = pt[(g + e) * kKeys + key];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
              const float4 t = *reinterpret_cast<const float4*>(tt + (u < n ? h + 4 * u : h) * nq + g);
              a[u] = fmaf(t.x, x[0], fmaf(t.y, x[1], fmaf(t.z, x[2], fmaf(t.w, x[3], a[u]))));
            }
          }
        }
        for (; g < nq; ++g) {
          const float x = pt[g * kKeys + key];
#pragma unroll
          for (int u = 0; u < 4; ++u)
            if (u < n) a[u] = fmaf(tt[(h + 4 * u) * nq + g], x, a[u]);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (u < n)
            *reinterpret_cast<bf16*>(wrow + slice<8>(h + 4 * u, key >> 3) + (key & 7) * 2) = __float2bfloat16(a[u]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int t = 0; t < kKeys / 16; ++t) {
      const int i = blk * (kKeys / 16) + t;
      cp_async_wait<kValueStages - 2>();
      __syncwarp();
      load(i + kValueStages - 1);
      if (mine && (b0 + blk) * kKeys + t * 16 < len) {
        uint32_t pa[4];
        ldmatrix_x4(pa[0], pa[1], pa[2], pa[3], wcur + slice<8>(head0 + (lane & 15), t * 2 + (lane >> 4)));
        const uint32_t va = ring + (i % kValueStages) * VT;
        const int row = (lane & 7) + (((lane >> 3) & 1) << 3), cb = lane >> 4;
#pragma unroll
        for (int jn = 0; jn < NC / 16; ++jn) {
          uint32_t v0, v1, v2, v3;
          ldmatrix_x4_trans(v0, v1, v2, v3, va + slice<C>(row, jn * 2 + cb));
          mma_bf16_16816(o[jn * 2], pa, v0, v1);
          mma_bf16_16816(o[jn * 2 + 1], pa, v2, v3);
        }
      }
      __syncwarp();
    }
  }
  cp_async_wait<0>();
  if (!mine) return;
  const int r0 = lane >> 2;
#pragma unroll
  for (int jn = 0; jn < NC / 8; ++jn) {
    const int c = col0 + jn * 8 + (lane & 3) * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = r0 + half * 8;
      if (r >= rows) continue;
      const float x = o[jn][half * 2], y = o[jn][half * 2 + 1];
      const int64_t head = (int64_t)b * nq + head0 + r;
      if (p.vsplits > 1) {
        *reinterpret_cast<float2*>(p.part + (head * p.vsplits + split) * D + c) = make_float2(x, y);
      } else {
        if (c < p.dv) p.out[head * p.dv + c] = __float2bfloat16(x);
        if (c + 1 < p.dv) p.out[head * p.dv + c + 1] = __float2bfloat16(y);
      }
    }
  }
}

__global__ void __launch_bounds__(128) talk_merge_kernel(bf16* __restrict__ out, const float* __restrict__ part, int splits, int dv) {
  const int64_t head = blockIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  const int c = threadIdx.x;
  if (c >= dv) return;
  float a = 0.f;
  for (int s = 0; s < splits; ++s) a += part[(head * splits + s) * D + c];
  out[head * dv + c] = __float2bfloat16(a);
}

// ------------------------------------------------------------------------------------------------ prompts
struct WeightsParams {
  const bf16* q;              // [total_q, nq, 128]
  const bf16* k_cache;
  const bf16* talk;
  const float* lse;           // [total_q, nq], log2 domain
  bf16* w;                    // [nq, w_rows, ld]
  const int32_t *block_table, *cu_q, *kv_lens;
  int64_t w_rows, ld;
  int bt_stride, nq, nkv, group, page, row0, rows, keys;   // keys: of a block, a multiple of 16
  SoftCap cap;
  float scale_log2;
};

constexpr int kUnits = 8, kBM = 16, kKStages = 3, kPairLine = 128;
constexpr int kPairBytes = kBM * 16 * kPairLine;      // pairs of one step

__device__ __forceinline__ int spread(int key) { return (key & 1) | ((key >> 1) & 2) | (((key >> 1 ^ key >> 3) & 1) << 2); }

// grid (tiles of 16 rows, ranges of keys, sequences), 8 warps.  HB: tiles of 16 heads; KS: tiles of 16 columns of T (two units each).
template <int HB, int KS>
__global__ void __launch_bounds__(256, 1) talk_weights_kernel(WeightsParams p) {
  extern __shared__ __align__(128) uint8_t smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  const int q_end = p.cu_q[b + 1], q_lo = max(p.cu_q[b], p.row0), q_hi = min(q_end, p.row0 + p.rows);
  const int tiles = q_hi > q_lo ? (q_hi - q_lo + kBM - 1) / kBM : 0;
  if ((int)blockIdx.x >= tiles) return;
  const int tile = tiles - 1 - blockIdx.x, r0 = q_lo + tile * kBM;                 // late tiles first
  const int kv_len = p.kv_lens[b], pos0 = kv_len - (q_end - r0);                   // position of row r0
  const int k0 = blockIdx.y * p.keys;
  // the product with the values takes tiles of 128 rows and of 128 keys: what their last row sees is defined for all of them
  const int big = q_lo + tile * kBM / 128 * 128;
  const int defined = (max(0, min(kv_len, kv_len - (q_end - big) + 128)) + 127) / 128 * 128;
  if (k0 >= defined) return;
  const int k_end = min(k0 + p.keys, defined);
  const int seen = min(kv_len, pos0 + min(kBM, q_hi - r0));                        // keys that some row of the tile sees
  const int steps = max(0, (min(k_end, seen) - k0 + 15) >> 4);
  const int subs = (p.group + 3) >> 2, units = p.nkv * subs;
  const bool mine = warp < units;
  const int kvh = mine ? warp / subs : 0, head0 = kvh * p.group + (mine ? (warp - kvh * subs) * 4 : 0);
  const int heads = mine ? min(4, kvh * p.group + p.group - head0) : 0;
  const uint32_t kring = smem_u32(smem);
  const int kbytes = p.nkv * kTileBytes;
  uint8_t* pair = smem + kKStages * kbytes;
  const uint32_t pair_u32 = smem_u32(pair);
  const int32_t* bt = p.block_table + (int64_t)b * p.bt_stride;

  const auto load = [&](int s) {                      // keys of step s of all kv heads
    if (s < steps) {
      const int tok0 = k0 + s * 16, pg = tok0 / p.page;
      const bf16* kb = p.k_cache + ((int64_t)bt[pg] * p.nkv * p.page + tok0 - pg * p.page) * D;
      const uint32_t dst = kring + (s % kKStages) * kbytes;
      for (int id = threadIdx.x; id < p.nkv * 16 * CH; id += 256) {
        const int c = id % CH, r = id / CH % 16, g = id / (16 * CH);
        const bool in = tok0 + r < kv_len;
        cp_async16(dst + g * kTileBytes + swz<CH>(r, c), kb + (in ? ((int64_t)g * p.page + r) * D + c * 8 : 0), in);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < kKStages - 1; ++s) load(s);
  if (units < 2 * KS)                                 // a chunk without a unit meets zeros of T and must be finite
    for (int i = threadIdx.x; i < 2 * kPairBytes / 16; i += 256) reinterpret_cast<uint4*>(pair)[i] = make_uint4(0, 0, 0, 0);

  // queries: B operand, columns are rows 0..7 and 8..15 of the tile
  uint32_t qf[4][2][16];
  float nl[4][2][2];                                  // minus the log-sum-exp of (head, row); -inf: no such pair
#pragma unroll
  for (int u = 0; u < 4; ++u)
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int row = r0 + n * 8 + (lane >> 2);
      const bool in = u < heads && row < q_hi;
      const bf16* src = p.q + ((int64_t)row * p.nq + head0 + u) * D + (lane & 3) * 2;
#pragma unroll
      for (int ks = 0; ks < 16; ++ks) qf[u][n][ks] = in ? *reinterpret_cast<const uint32_t*>(src + ks * 8) : 0u;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = r0 + n * 8 + (lane & 3) * 2 + e;
        nl[u][n][e] = u < heads && r < q_hi ? -p.lse[(int64_t)r * p.nq + head0 + u] : -INFINITY;
      }
    }
  // T: A operand, columns: unit by unit four leading terms, four remainders
  uint32_t ta[HB][KS][4];
#pragma unroll
  for (int hb = 0; hb < HB; ++hb)
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int h = hb * 16 + (lane >> 2) + (i & 1) * 8, u = (lane & 1) * 2, un = ks * 2 + (i >> 1);
        const int c = un / subs, first = (un - c * subs) * 4;
        const bf16 zero = __float2bfloat16(0.f);
        const auto at = [&](int e) {
          return h < p.nq && un < units && first + u + e < p.group ? p.talk[h * p.nq + c * p.group + first + u + e] : zero;
        };
        const bf162 v = __halves2bfloat162(at(0), at(1));
        ta[hb][ks][i] = *reinterpret_cast<const uint32_t*>(&v);
      }

  const auto scores = [&](int s) {
    const uint32_t ka = kring + (s % kKStages) * kbytes + kvh * kTileBytes;
    float x[4][2][4];
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
      for (int n = 0; n < 2; ++n) x[u][n][0] = x[u][n][1] = x[u][n][2] = x[u][n][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 8; ++ks) {
      uint32_t a[4];
      ldmatrix_x4(a[0], a[1], a[2], a[3], ka + swz<CH>(lane & 15, ks * 2 + (lane >> 4)));
#pragma unroll
      for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int n = 0; n < 2; ++n) mma_bf16_16816(x[u][n], a, qf[u][n][ks * 2], qf[u][n][ks * 2 + 1]);
    }
    const int key0 = k0 + s * 16;
    const bool edge = key0 + 15 > pos0;               // some row does not see all of these keys
    const uint32_t dst = pair_u32 + (s & 1) * kPairBytes;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int key = (lane >> 2) + (j >> 1) * 8, r = n * 8 + (lane & 3) * 2 + (j & 1);
        float f[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) f[u] = exp2f(score(x[u][n][j], p.cap, p.scale_log2) + nl[u][n][j & 1]);
        if (edge && key0 + key > pos0 + r) f[0] = f[1] = f[2] = f[3] = 0.f;
        uint32_t hi[2], lo[2];
        split_pack(f[0], f[1], hi[0], lo[0]);
        split_pack(f[2], f[3], hi[1], lo[1]);
        const uint32_t at = dst + (r * 16 + key) * kPairLine + ((warp ^ spread(key)) << 4);
        asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(at), "r"(hi[0]), "r"(hi[1]), "r"(lo[0]), "r"(lo[1]) : "memory");
      }
  };
  const auto mix = [&](int s) {
    const uint32_t src = pair_u32 + (s & 1) * kPairBytes;
    const int n = lane & 7, mi = lane >> 3, key = 4 * (n >> 1) + (n & 1) + (mi >> 1) * 2;     // this lane's line
#pragma unroll
    for (int i = 0; i < kBM / 8; ++i) {
      const int r = warp + 8 * i;
      float d[HB][2][4];
#pragma unroll
      for (int hb = 0; hb < HB; ++hb)
#pragma unroll
        for (int t = 0; t < 2; ++t) d[hb][t][0] = d[hb][t][1] = d[hb][t][2] = d[hb][t][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, src + (r * 16 + key) * kPairLine + (((ks * 2 + (mi & 1)) ^ spread(key)) << 4));
#pragma unroll
        for (int hb = 0; hb < HB; ++hb) {
          mma_bf16_16816(d[hb][0], ta[hb][ks], b0, b1);
          mma_bf16_16816(d[hb][1], ta[hb][ks], b2, b3);
        }
      }
      if (r0 + r >= q_hi) continue;
      bf16* dst = p.w + (int64_t)(r0 + r - p.row0) * p.ld + k0 + s * 16 + 4 * (lane & 3);
#pragma unroll
      for (int hb = 0; hb < HB; ++hb)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int h = hb * 16 + (lane >> 2) + half * 8;
          if (h < p.nq)
            *reinterpret_cast<uint2*>(dst + (int64_t)h * p.w_rows * p.ld) =
                make_uint2(pack_bf162(d[hb][0][half * 2], d[hb][0][half * 2 + 1]), pack_bf162(d[hb][1][half * 2], d[hb][1][half * 2 + 1]));
        }
    }
  };
  for (int s = 0; s < steps; ++s) {
    cp_async_wait<kKStages - 2>();
    __syncthreads();                                  // keys of step s are here; step s - 1's weights are; step s - 2's mixture is done
    load(s + kKStages - 1);
    if (mine) scores(s);
    if (s > 0) mix(s - 1);
  }
  cp_async_wait<0>();
  __syncthreads();
  if (steps > 0) mix(steps - 1);
  // keys that no row of the tile sees
  const int z0 = k0 + steps * 16, per = (k_end - z0) / 8;
  for (int i = threadIdx.x; per > 0 && i < p.nq * kBM * per; i += 256) {
    const int c = i % per, r = i / per % kBM, h = i / (per * kBM);
    if (r0 + r < q_hi)
      *reinterpret_cast<uint4*>(p.w + ((int64_t)h * p.w_rows + r0 + r - p.row0) * p.ld + z0 + c * 8) = make_uint4(0, 0, 0, 0);
  }
}

template <typename K>
static int prepare(K kernel, size_t smem) {
  // the largest size seen; a race of two first calls sets the same attribute twice
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

}  // namespace talk
}  // namespace xllm

// fp32 elements of workspace xllm_talk_decode needs.
XLLM_API int64_t xllm_talk_decode_workspace(int64_t batch, int nq, int64_t ld, int splits, int vsplits) {
  return batch * nq * (ld + 2 * (int64_t)splits + (vsplits > 1 ? (int64_t)vsplits * xllm::talk::D : 0));
}

// out [B, nq, dv] of one query row per sequence, q [B, nq, 128], caches [n_blocks, nkv, page, 128], talk [nq, nq]; seq_lens [B];
// ld: an even number of scores a row may have, a multiple of 16 no less than the longest sequence; page % 16 == 0; nq <= 64.
XLLM_API int xllm_talk_decode(void* out, const void* q, const void* k_cache, const void* v_cache, const void* talk_w,
                              const void* block_table, int bt_stride, const void* seq_lens, int batch, int nq, int nkv, int dv, int page,
                              float scale, float softcap, int64_t ld, int splits, int vsplits, void* workspace, void* stream) {
  using namespace xllm;
  using namespace xllm::talk;
  if (batch == 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv || nq > kMaxHeads || dv <= 0 || dv > D || page <= 0 || page % 16 || ld <= 0 || ld % 16 || splits < 1 ||
      vsplits < 1 || workspace == nullptr || (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)workspace) & 15))
    return (int)cudaErrorInvalidValue;
  DecodeParams p;
  p.q = (const bf16*)q; p.k_cache = (const bf16*)k_cache; p.v_cache = (const bf16*)v_cache; p.talk = (const bf16*)talk_w;
  p.out = (bf16*)out; p.s = (float*)workspace; p.stat = (float2*)(p.s + (int64_t)batch * nq * ld);
  p.part = (float*)(p.stat + (int64_t)batch * nq * splits); p.block_table = (const int32_t*)block_table;
  p.seq_lens = (const int32_t*)seq_lens; p.ld = ld; p.bt_stride = bt_stride; p.nq = nq; p.nkv = nkv; p.group = nq / nkv; p.page = page;
  p.splits = splits; p.vsplits = vsplits; p.dv = dv; p.cap = make_soft_cap(scale, softcap); p.scale_log2 = scale * kLog2e;
  cudaStream_t s = (cudaStream_t)stream;
  const int qtiles = (p.group + 15) / 16, units = nkv * qtiles;
  const size_t smem1 = 4 * kScoreStages * kTileBytes;
  const int wpu = units >= 8 ? 1 : (units >= 4 ? 2 : (units >= 2 ? 4 : 8));
  const size_t smem2 = (size_t)8 * kValueStages * 16 * (D / wpu) * 2 + (size_t)2 * (nq + 16) * kKeys * 2 +
                       ((size_t)nq * kKeys + (size_t)nq * nq + nq) * 4;
  int rc = prepare(talk_scores_tc_kernel, smem1);
  if (rc != 0) return rc;
  launch_pdl(talk_scores_tc_kernel, dim3(units, batch, splits), dim3(128), smem1, s, p);
  const dim3 grid((units * wpu + 7) / 8, batch, vsplits);
  const auto run = [&](auto kernel) {
    const int e = prepare(kernel, smem2);
    if (e == 0) launch_pdl(kernel, grid, dim3(256), smem2, s, p);
    return e;
  };
  rc = wpu == 1 ? run(talk_decode_kernel<1>) : (wpu == 2 ? run(talk_decode_kernel<2>) : (wpu == 4 ? run(talk_decode_kernel<4>) : run(talk_decode_kernel<8>)));
  if (rc != 0) return rc;
  if (vsplits > 1)
    launch_pdl(talk_merge_kernel, dim3((unsigned)((int64_t)batch * nq)), dim3(128), 0, s, p.out, (const float*)p.part, vsplits, dv);
  return XLLM_LAUNCH_CHECK();
}

// Mixed weights of the rows [row0, row0 + rows) of all sequences to w [nq, w_rows, ld] bf16 (see xllm_talk_values_tc), from q
// [total_q, nq, 128], the K cache and lse [total_q, nq] (xllm_prefill_lse_tc).  ld a multiple of 128 no less than the longest sequence;
// page % 16 == 0; no more than eight units of four heads of one key/value head.
XLLM_API int xllm_talk_weights(void* w, int64_t w_rows, int64_t ld, const void* q, const void* k_cache, const void* talk_w, const void* lse,
                               const void* block_table, int bt_stride, const void* cu_q, const void* kv_lens, int batch, int max_q_len,
                               int row0, int rows, int nq, int nkv, int page, float scale, float softcap, int keys, void* stream) {
  using namespace xllm;
  using namespace xllm::talk;
  if (batch == 0 || rows == 0 || max_q_len == 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv || page <= 0 || page % 16 || ld <= 0 || ld % 128 || w_rows < rows || keys <= 0 || keys % 128 ||
      (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)w) & 15))
    return (int)cudaErrorInvalidValue;
  const int units = nkv * ((nq / nkv + 3) / 4);
  if (units > kUnits) return (int)cudaErrorInvalidValue;
  WeightsParams p;
  p.q = (const bf16*)q; p.k_cache = (const bf16*)k_cache; p.talk = (const bf16*)talk_w; p.lse = (const float*)lse; p.w = (bf16*)w;
  p.block_table = (const int32_t*)block_table; p.cu_q = (const int32_t*)cu_q; p.kv_lens = (const int32_t*)kv_lens; p.w_rows = w_rows;
  p.ld = ld; p.bt_stride = bt_stride; p.nq = nq; p.nkv = nkv; p.group = nq / nkv; p.page = page; p.row0 = row0; p.rows = rows;
  p.keys = keys; p.cap = make_soft_cap(scale, softcap); p.scale_log2 = scale * kLog2e;
  const dim3 grid((unsigned)((min(max_q_len, rows) + kBM - 1) / kBM), (unsigned)((ld + keys - 1) / keys), batch);
  const size_t smem = (size_t)kKStages * nkv * kTileBytes + 2 * kPairBytes;
  const auto run = [&](auto kernel) {
    const int e = prepare(kernel, smem);
    if (e != 0) return e;
    launch_pdl(kernel, grid, dim3(256), smem, (cudaStream_t)stream, p);
    return XLLM_LAUNCH_CHECK();
  };
  if (nq <= 16) {
    if (units <= 2) return run(talk_weights_kernel<1, 1>);
    if (units <= 4) return run(talk_weights_kernel<1, 2>);
    return run(talk_weights_kernel<1, 4>);
  }
  return run(talk_weights_kernel<2, 4>);
}
