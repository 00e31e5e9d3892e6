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
// The mixture of 16 rows, 128 keys at a time.  tcgen05 products leave transposed scores in tensor memory: a lane per key, and per unit
// (up to four heads of one key/value head) row by row its heads.  So a thread has the weights of a unit for a pair at once and stores
// them as one 16-byte chunk of the pair's line: four leading terms, four remainders.  The lines of a row are the B operand of its
// mixture (mma.sync m16n8k16, pairs as N, chunks as K), T repeated for leading terms and remainders the A operand, and what comes out
// is four neighbouring keys per thread.  A row's mixture is computed beside the next row's exponentials.  Every mbarrier wait is
// bounded; on expiry all roles leave, tensor memory is released and an error word is set (xllm_talk_error_status).
#include "attn_common.cuh"
#include "tc_common.cuh"
#include <type_traits>

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
  const bf16* talk;
  const float* lse;           // [total_q, nq], log2 domain
  bf16* w;                    // [nq, w_rows, ld]
  const int32_t *block_table, *cu_q, *kv_lens;
  int64_t w_rows, ld;
  int bt_stride, nq, nkv, group, page_log2, row0, rows, keys;   // keys: of a block, a multiple of 16
  SoftCap cap;
  float scale_log2;
  int* err;
};
static int* g_err[64] = {};

constexpr int kUnits = 8, kBM = 16, kBN = 128;        // rows of a CTA, keys of a tile
constexpr int kUnitCols = 4 * kBM;                    // scores of a key: row by row four heads
constexpr int kQUnit = kUnitCols * D * 2;             // bytes of a unit's queries
constexpr int kKTile = kBN * D * 2, kHalf = kKTile / 2;
constexpr int kLine = 128, kLines = kBN * kLine;      // weights of a pair, of a row's pairs in one tile
constexpr int kWorkers = 16, kThreads = (kWorkers + 2) * 32;
constexpr int kNlOff = kUnits * kQUnit + 2 * kKTile + 2 * kLines, kBarOff = kNlOff + kBM * kUnits * 4 * 4;
constexpr int kWeightsSmem = kBarOff + (1 + 4 + 2 * kUnits) * 8 + 16;     // no slack: the block's limit is near

// The line of a pair keeps chunk c at c ^ spread(key): eight neighbouring keys (stores) and the eight keys of half an operand (loads)
// meet eight different places.
__device__ __forceinline__ int spread(int key) { return (key & 1) | ((key >> 1) & 2) | (((key >> 1 ^ key >> 3) & 1) << 2); }

// Pairs of fp32 values in one instruction.
__device__ __forceinline__ uint64_t pack2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2f(uint64_t v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// Two weights from their scores; CAP: 0 none, 1 the polynomial, 2 any score.
template <int CAP>
__device__ __forceinline__ void weigh(const uint32_t* x, uint64_t nl, const uint64_t (&k)[4], const SoftCap& cap, float& f0, float& f1) {
  const float x0 = __uint_as_float(x[0]), x1 = __uint_as_float(x[1]);
  if constexpr (CAP == 2) {
    unpack2f(add2(pack2(soft_cap(x0, cap), soft_cap(x1, cap)), nl), f0, f1);
  } else {
    const uint64_t v = pack2(x0, x1);
    if constexpr (CAP == 1) {
      const uint64_t v2 = mul2(v, v);
      unpack2f(fma2(v, fma2(v2, fma2(v2, fma2(v2, k[3], k[2]), k[1]), k[0]), nl), f0, f1);
    } else {
      unpack2f(fma2(v, k[0], nl), f0, f1);
    }
  }
  f0 = exp2f(f0);
  f1 = exp2f(f1);
}

// The chunk of one unit's four heads: the weights rounded to bf16, and what that left.
template <int CAP, bool EDGE>
__device__ __forceinline__ void chunk_out(uint32_t at, const uint32_t* x, uint32_t nl_at, const uint64_t (&k)[4], const SoftCap& cap,
                                          bool hidden) {
  uint64_t nl[2];
  asm volatile("ld.shared.v2.b64 {%0, %1}, [%2];" : "=l"(nl[0]), "=l"(nl[1]) : "r"(nl_at));
  uint32_t hi[2], lo[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    float f0, f1, r0, r1;
    weigh<CAP>(x + 2 * i, nl[i], k, cap, f0, f1);
    if (EDGE && hidden) f0 = f1 = 0.f;
    hi[i] = pack_bf162(f0, f1);
    asm("{.reg .b16 a, b; mov.b32 {a, b}, %2; sub.rn.f32.bf16 %0, a, %3; sub.rn.f32.bf16 %1, b, %4;}"
        : "=f"(r0), "=f"(r1)
        : "r"(hi[i]), "f"(f0), "f"(f1));
    lo[i] = pack_bf162(-r0, -r1);
  }
  asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(at), "r"(hi[0]), "r"(hi[1]), "r"(lo[0]), "r"(lo[1]) : "memory");
}

// grid (tiles of 16 rows, ranges of keys, sequences).  Warps 0-15: worker w has keys 32 (w % 4) .. + 31 of a tile for units 2 (w / 4)
// and the next, and mixes keys 16 (w % 8) .. + 15 for heads 16 (w / 8) .. + 15; warp 16 loads, warp 17 issues the products.  KS: tiles
// of 16 columns of T (two units each).
template <int KS>
__global__ void __launch_bounds__(kThreads, 1)
talk_weights_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k, const __grid_constant__ WeightsParams p) {
  using namespace tc;
  extern __shared__ __align__(1024) uint8_t smem[];
  const auto nl = reinterpret_cast<float(*)[kUnits * 4]>(smem + kNlOff);  // minus the log-sum-exps; -inf: no such pair
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(smem + kBarOff + (1 + 4 + 2 * kUnits) * 8);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z;
  const int q_end = p.cu_q[b + 1], q_lo = max(p.cu_q[b], p.row0), q_hi = min(q_end, p.row0 + p.rows);
  const int tiles = q_hi > q_lo ? (q_hi - q_lo + kBM - 1) / kBM : 0;
  if ((int)blockIdx.x >= tiles) return;               // uniform for the whole CTA: nothing allocated yet
  const int tile = tiles - 1 - blockIdx.x, r0 = q_lo + tile * kBM;                 // late tiles first
  const int kv_len = p.kv_lens[b], pos0 = kv_len - (q_end - r0);                   // position of row r0
  const int k0 = blockIdx.y * p.keys;
  // the product with the values takes tiles of 128 rows: what their last row sees, rounded up, is defined for all of them
  const int big = q_lo + tile * kBM / 128 * 128;
  const int defined = (max(0, min(kv_len, kv_len - (q_end - big) + 128)) + 127) / 128 * 128;
  if (k0 >= defined) return;
  const int k_end = min(k0 + p.keys, defined);
  const int seen = min(kv_len, pos0 + min(kBM, q_hi - r0));                        // keys that some row of the tile sees
  const int n = max(0, (min(k_end, seen) - k0 + kBN - 1) / kBN);                   // key tiles
  const int subs = (p.group + 3) >> 2, units = p.nkv * subs;
  const auto head_of = [&](int unit) { return unit / subs * p.group + unit % subs * 4; };
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  const uint32_t sbase = smem_u32(smem);
  if (sbase & 1023) {                                 // swizzled tiles need the alignment asked for above
    if (threadIdx.x == 0 && p.err != nullptr) atomicExch(p.err, 2);
    return;
  }
  const uint32_t qsm = sbase, ksm = qsm + kUnits * kQUnit, lines = ksm + 2 * kKTile;
  const uint32_t bar0 = sbase + kBarOff, q_full = bar0;
  const auto k_full = [&](int s) { return bar0 + 8u * (1 + s); };
  const auto k_empty = [&](int s) { return bar0 + 8u * (3 + s); };
  const auto s_full = [&](int u) { return bar0 + 8u * (5 + u); };
  const auto s_free = [&](int u) { return bar0 + 8u * (5 + kUnits + u); };

  if (n > 0) {
    if (threadIdx.x == 0) {
      mbar_init(q_full, 1);
      for (int s = 0; s < 2; ++s) {
        mbar_init(k_full(s), 1);
        mbar_init(k_empty(s), 1);
      }
      for (int u = 0; u < kUnits; ++u) {
        mbar_init(s_full(u), 1);
        mbar_init(s_free(u), 4);
      }
      *abort_flag = 0;
      asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == kWorkers + 1) {
      asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_holder)), "r"(512));
      asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
    }
    for (int i = threadIdx.x; i < kBM * kUnits * 4; i += kThreads) {
      const int r = i / (kUnits * 4), c = i % (kUnits * 4), unit = c >> 2, u = c & 3;
      const bool in = unit < units && unit % subs * 4 + u < p.group && r0 + r < q_hi;
      nl[r][c] = in ? -p.lse[(int64_t)(r0 + r) * p.nq + head_of(unit) + u] : -INFINITY;
    }
    for (int i = threadIdx.x; i < 2 * kLines / 16; i += kThreads)      // chunks without a unit meet zeros of T and must be finite
      asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};" ::"r"(lines + i * 16), "r"(0) : "memory");
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_holder;

    if (warp == kWorkers) {
      // ---------------------------------------------------------------- loads
      if (lane == 0) {
        mbar_expect_tx(q_full, units * kQUnit);
        for (int u = 0; u < units; ++u)
          for (int h = 0; h < 2; ++h) tma_load_3d(qsm + u * kQUnit + h * (kQUnit / 2), &tma_q, h * 64, head_of(u), r0, q_full);
      }
      __syncwarp();
      const int page = 1 << p.page_log2, pages = kBN >> p.page_log2, n_blk = (kv_len + page - 1) >> p.page_log2;
      const int32_t* bt = p.block_table + (int64_t)b * p.bt_stride;
      bool ok = true;
      for (int t = 0, i = 0; t < n && ok; ++t) {
        const int pg = ((k0 + t * kBN) >> p.page_log2) + lane;
        const int blk = lane < pages && pg < n_blk ? bt[pg] : 0;       // pages past the sequence read block 0 (hidden)
        for (int c = 0; c < p.nkv; ++c, ++i) {
          const int st = i & 1;
          if (!mbar_wait_warp(k_empty(st), ((i >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
          if (lane == 0) mbar_expect_tx(k_full(st), kKTile);
          __syncwarp();
          if (lane < pages) {
            const uint32_t dst = ksm + st * kKTile + lane * page * 128;
            const int y = (blk * p.nkv + c) << p.page_log2;
            tma_load_2d(dst, &tma_k, 0, y, k_full(st));
            tma_load_2d(dst + kHalf, &tma_k, 64, y, k_full(st));
          }
          __syncwarp();
        }
      }
      if (!ok) {
        const long long t0 = clock64();
        while (clock64() - t0 < 20000000LL) {}        // bounded grace period for copies in flight
      }
    } else if (warp == kWorkers + 1) {
      // ---------------------------------------------------------------- products: [128 keys] x [16 rows x 4 heads] per unit
      constexpr uint32_t ID = idesc(false, kUnitCols);
      bool ok = mbar_wait_warp(q_full, 0, abort_flag);
      for (int t = 0, i = 0; t < n && ok; ++t)
        for (int c = 0; c < p.nkv && ok; ++c, ++i) {
          const int st = i & 1;
          ok = mbar_wait_warp(k_full(st), (i >> 1) & 1, abort_flag);
          for (int j = 0; j < subs && ok; ++j) {
            const int u = c * subs + j;
            ok = mbar_wait_warp(s_free(u), (t & 1) ^ 1, abort_flag);
            if (!ok) break;
            tc_fence_after();
            if (lane == 0) {
              const uint32_t ka = ksm + st * kKTile, qa = qsm + u * kQUnit;
#pragma unroll
              for (int ks = 0; ks < 8; ++ks)
                umma(tmem + u * kUnitCols, smem_desc(ka + (ks >> 2) * kHalf + (ks & 3) * 32, 16, 1024),
                     smem_desc(qa + (ks >> 2) * (kQUnit / 2) + (ks & 3) * 32, 16, 1024), ID, ks != 0);
              if (j == subs - 1 && i + 2 < n * p.nkv) umma_commit(k_empty(st));
              umma_commit(s_full(u));
            }
            __syncwarp();
          }
        }
    } else {
      // ---------------------------------------------------------------- weights and their mixture
      const int quarter = warp & 3, u0 = (warp >> 2) * 2, key = quarter * 32 + lane;
      const int hb = warp >> 3, kb = (warp & 7) * 16;
      const bool mixes = hb * 16 < p.nq;
      uint64_t k[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) k[i] = pack2(p.cap.k[i], p.cap.k[i]);
      if (!(p.cap.out > 0.f)) k[0] = pack2(p.scale_log2, p.scale_log2);
      // T: A operand, columns: unit by unit four leading terms, four remainders
      uint32_t ta[KS][4];
#pragma unroll
      for (int ks = 0; ks < KS; ++ks)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int h = hb * 16 + (lane >> 2) + (i & 1) * 8, u = (lane & 1) * 2, un = ks * 2 + (i >> 1), first = un % subs * 4 + u;
          const bf16 zero = __float2bfloat16(0.f);
          const auto at = [&](int e) { return h < p.nq && un < units && first + e < p.group ? p.talk[h * p.nq + head_of(un) + u + e] : zero; };
          const bf162 v = __halves2bfloat162(at(0), at(1));
          ta[ks][i] = *reinterpret_cast<const uint32_t*>(&v);
        }
      uint32_t chunk[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) chunk[j] = lines + key * kLine + (((u0 + j) ^ spread(key & 15)) << 4);
      const int mi = lane >> 3, mkey = 4 * ((lane & 7) >> 1) + (lane & 1) + (mi >> 1) * 2;
      uint32_t line[KS];                              // of row 0, by tile of T's columns
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) line[ks] = lines + (kb + mkey) * kLine + (((ks * 2 + (mi & 1)) ^ spread(mkey)) << 4);
      const uint32_t nl_at = sbase + kNlOff + u0 * 16;
      const uint32_t taddr = tmem + ((uint32_t)(quarter * 32) << 16) + u0 * kUnitCols;
      // place of (head hb 16 + lane / 4, row 0, key kb + 4 (lane % 4)) in the table
      const uint32_t place = (uint32_t)(((int64_t)(hb * 16 + (lane >> 2)) * p.w_rows + r0 - p.row0) * p.ld + k0 + kb + 4 * (lane & 3));
      const uint32_t heads8 = (uint32_t)(8 * p.w_rows * p.ld), ld = (uint32_t)p.ld;
      const bool h0 = hb * 16 + (lane >> 2) < p.nq, h1 = hb * 16 + 8 + (lane >> 2) < p.nq;
      const int rows = min(kBM, q_hi - r0);
      bool ok = true;

      const auto mix = [&](int t, int r) {            // row r of tile t
        if (!mixes) return;
        float d[2][4];
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(b0, b1, b2, b3, line[ks] + (r & 1) * kLines);
          if (ks == 0) {
            mma_bf16_16816_first(d[0], ta[0], b0, b1);
            mma_bf16_16816_first(d[1], ta[0], b2, b3);
          } else {
            mma_bf16_16816(d[0], ta[ks], b0, b1);
            mma_bf16_16816(d[1], ta[ks], b2, b3);
          }
        }
        if (r >= rows) return;
        const uint32_t at = place + r * ld + t * kBN;
        if (h0) *reinterpret_cast<uint2*>(p.w + at) = make_uint2(pack_bf162(d[0][0], d[0][1]), pack_bf162(d[1][0], d[1][1]));
        if (h1) *reinterpret_cast<uint2*>(p.w + at + heads8) = make_uint2(pack_bf162(d[0][2], d[0][3]), pack_bf162(d[1][2], d[1][3]));
      };
      for (int t = 0; t < n; ++t) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
          if (u0 + j < units) ok = ok && mbar_wait_warp(s_full(u0 + j), t & 1, abort_flag);
        tc_fence_after();
        const int late = k0 + t * kBN + key - pos0;   // rows before it do not see the key
        const bool edge = k0 + t * kBN + kBN - 1 > pos0;
#pragma unroll 1
        for (int q = 0; q < kBM / 4; ++q) {           // four rows from tensor memory at a time
          uint32_t x[2][16];
          float top = 0.f;
#pragma unroll
          for (int j = 0; j < 2; ++j)
            if (u0 + j < units) tmem_ld16(taddr + j * kUnitCols + q * 16, x[j]);
          tmem_ld_wait();
          if (q == kBM / 4 - 1) {                     // the next tile's products may overwrite the scores
            tc_fence_before();
            __syncwarp();
            if (lane == 0) {
#pragma unroll
              for (int j = 0; j < 2; ++j)
                if (u0 + j < units) mbar_arrive(s_free(u0 + j));
            }
          }
          if (p.cap.out > 0.f) {
#pragma unroll
            for (int j = 0; j < 2; ++j)
              if (u0 + j < units) {
#pragma unroll
                for (int i = 0; i < 16; i += 2)
                  asm("{.reg .f32 a, b; abs.f32 a, %1; abs.f32 b, %2; max.f32 %0, %0, a, b;}"
                      : "+f"(top)
                      : "f"(__uint_as_float(x[j][i])), "f"(__uint_as_float(x[j][i + 1])));
              }
          }
          const auto four_rows = [&](auto cap, auto edge) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int r = q * 4 + e;
              // the row before: its lines are complete since the last barrier
              if (r > 0) mix(t, r - 1);
              else if (t > 0) mix(t - 1, kBM - 1);
#pragma unroll
              for (int j = 0; j < 2; ++j)
                if (u0 + j < units)
                  chunk_out<decltype(cap)::value, decltype(edge)::value>(chunk[j] + (e & 1) * kLines, x[j] + e * 4,
                                                                         nl_at + (r * kUnits + j) * 16, k, p.cap, late > r);
              asm volatile("bar.sync 1, 512;" ::: "memory");
            }
          };
          using std::integral_constant;
          if (!(p.cap.out > 0.f)) four_rows(integral_constant<int, 0>(), std::true_type());
          else if (!__all_sync(0xffffffffu, top <= p.cap.small)) four_rows(integral_constant<int, 2>(), std::true_type());
          else if (edge) four_rows(integral_constant<int, 1>(), std::true_type());
          else four_rows(integral_constant<int, 1>(), std::false_type());
        }
      }
      mix(n - 1, kBM - 1);
    }
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0 && *abort_flag && p.err != nullptr) atomicExch(p.err, 1);
    if (warp == kWorkers + 1) {
      tc_fence_after();
      asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512));
    }
  }
  // keys that no row of the tile sees
  const int z0 = k0 + n * kBN, per = (k_end - z0) / 8;
  for (int i = threadIdx.x; per > 0 && i < p.nq * kBM * per; i += kThreads) {
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
// page 16, 32, 64 or 128; no more than eight units of four heads of one key/value head, nor 32 heads.
XLLM_API int xllm_talk_weights(void* w, int64_t w_rows, int64_t ld, const void* q, int64_t total_q, const void* k_cache, int64_t n_blocks,
                               const void* talk_w, const void* lse,
                               const void* block_table, int bt_stride, const void* cu_q, const void* kv_lens, int batch, int max_q_len,
                               int row0, int rows, int nq, int nkv, int page, float scale, float softcap, int keys, void* stream) {
  using namespace xllm;
  using namespace xllm::talk;
  if (batch == 0 || rows == 0 || max_q_len == 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv || nq > 32 || page < 16 || page > 128 || (page & (page - 1)) || ld <= 0 || ld % 128 || w_rows < rows || keys <= 0 || keys % 128 ||
      (int64_t)nq * w_rows * ld >= (1LL << 32) ||
      (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)w) & 15))
    return (int)cudaErrorInvalidValue;
  const int units = nkv * ((nq / nkv + 3) / 4);
  if (units > kUnits) return (int)cudaErrorInvalidValue;
  WeightsParams p{};
  p.talk = (const bf16*)talk_w; p.lse = (const float*)lse; p.w = (bf16*)w;
  p.block_table = (const int32_t*)block_table; p.cu_q = (const int32_t*)cu_q; p.kv_lens = (const int32_t*)kv_lens; p.w_rows = w_rows;
  p.ld = ld; p.bt_stride = bt_stride; p.nq = nq; p.nkv = nkv; p.group = nq / nkv; p.row0 = row0; p.rows = rows;
  while ((16 << p.page_log2) < page) ++p.page_log2;
  p.page_log2 += 4;
  p.keys = keys; p.cap = make_soft_cap(scale, softcap); p.scale_log2 = scale * kLog2e;
  const dim3 grid((unsigned)((min(max_q_len, rows) + kBM - 1) / kBM), (unsigned)((ld + keys - 1) / keys), batch);
  int dev = 0;
  cudaGetDevice(&dev);
  if (g_err[dev & 63] == nullptr) {
    if (cudaMalloc(&g_err[dev & 63], sizeof(int)) != cudaSuccess) return (int)cudaErrorMemoryAllocation;
    cudaMemset(g_err[dev & 63], 0, sizeof(int));
  }
  p.err = g_err[dev & 63];
  CUtensorMap tq, tk;
  if (!tc::make_map_heads(&tq, q, total_q, nq, kBM, 4) || !tc::make_map(&tk, k_cache, n_blocks * nkv * page, D, D, page))
    return (int)cudaErrorInvalidValue;
  const auto run = [&](auto kernel) {
    const int e = prepare(kernel, kWeightsSmem);
    if (e != 0) return e;
    kernel<<<grid, kThreads, kWeightsSmem, (cudaStream_t)stream>>>(tq, tk, p);
    return XLLM_LAUNCH_CHECK();
  };
  return units <= 2 ? run(talk_weights_kernel<1>) : (units <= 4 ? run(talk_weights_kernel<2>) : run(talk_weights_kernel<4>));
}

// 0 = no bounded wait expired in the prompt kernel on this device since the last call.
XLLM_API int xllm_talk_error_status() {
  int dev = 0, v = 0;
  cudaGetDevice(&dev);
  int* e = xllm::talk::g_err[dev & 63];
  if (e == nullptr) return 0;
  cudaMemcpy(&v, e, sizeof(int), cudaMemcpyDeviceToHost);
  if (v != 0) cudaMemset(e, 0, sizeof(int));
  return v;
}
