// Varlen causal prefill attention over the paged KV cache on the 5th-generation tensor cores.
//
// One CTA = (sequence, query head, tile of 128 query tokens), head_dim 128, 320 threads:
//   warp 0      TMA producer: the Q tile once, then K and V tiles of 128 tokens into a two-stage
//               shared-memory ring; a tile is gathered page by page through the block table (one
//               [page x 64]-element box per page and half of the head dimension)
//   warp 1      MMA issuer: S = Q K^T (tcgen05.mma, both operands K-major) into one of two S
//               accumulators in TMEM; then, once the softmax warps have written P, O_tile = P V
//               with V as an MN-major operand (the cache keeps head_dim contiguous), into one of two
//               O accumulators.  QK of tile j+1 is issued before PV of tile j, so the tensor pipe
//               works while the softmax of tile j runs.
//   warps 2-9   softmax: two threads per query row, 64 columns each (tcgen05.ld gives a thread its
//               own row; the two halves exchange their row maximum through shared memory); P goes to
//               shared memory as bf16 in the 128-byte swizzled K-major layout; the finished O tile
//               of the previous step is added with the usual rescaling O = (O + O_tile) * alpha.
// The reference reaches the same op through FlashInfer's fa2 kernels
// (xllm/core/kernels/cuda/flashinfer_attention.cpp:239-301); the mma.sync kernel of attn_prefill.cu
// stays as the path for other head sizes and small pages.
//
// Every mbarrier wait is bounded; on expiry all roles leave, TMEM is released and an error word
// is set (xllm_fmha_error_status).
#include "attn_common.cuh"
#include "tc_common.cuh"

namespace xllm {
namespace fmha {

using namespace tc;

constexpr int kD = 128;
constexpr int kBM = 128;  // query rows per CTA
constexpr int kBN = 128;  // kv tokens per tile
constexpr int kHalf = kBM * 128;          // bytes of one [128 rows x 64 elements] swizzled half tile
constexpr int kTile = 2 * kHalf;          // 32 KB: a [128 x 128] bf16 operand tile

constexpr int Q_OFF = 0;
constexpr int KV_OFF = kTile;                       // 2 stages x (K, V)
constexpr int P_OFF = KV_OFF + 4 * kTile;
constexpr int BAR_OFF = P_OFF + kTile;
constexpr int XCH_OFF = BAR_OFF + 24 * 8 + 16;          // row-max / row-sum exchange between the two halves of a row
constexpr int SMEM_TOTAL = XCH_OFF + (2 * 2 + 2) * kBM * 4 + 1024;
constexpr int LSE_CUT = 3 * kTile;                  // what a CTA without values and weights does not need: two of them fit an SM

struct Params {
  bf16* out;
  const int32_t* block_table;
  const int32_t* cu_q;
  const int32_t* kv_lens;
  int64_t o_stride;
  int bt_stride, nq, nkv, page, causal;
  int window;                  // > 0: a query sees its last `window` positions only
  int keep;                    // ... and the first `keep`
  int rows_kv;                 // K and V are rows of all heads (page n: rows n * page ..), not one tile per page and head
  SoftCap cap;
  float scale_log2;
  int* err;
  const float* sink;           // [nq] a score per head that joins the denominator, or null
  float* lse;                  // optional [total_q, nq]: log2-domain log-sum-exp of every row's scaled scores
};

// LSE: nothing but the log-sum-exp of every row (no values, no output).
template <bool CAP, bool LSE>
__global__ void __launch_bounds__(320, LSE ? 2 : 1)
prefill_tc_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                  const __grid_constant__ CUtensorMap tma_v, const Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  constexpr int CUT = LSE ? LSE_CUT : 0, KV_STAGE = LSE ? kTile : 2 * kTile, TMEM_COLS = LSE ? 256 : 512;
  const uint32_t bar0 = sbase + BAR_OFF - CUT;
  // barrier slots
  // K and V have rings of their own: a K slot is free again as soon as the QK product that read it
  // has completed, a V slot after its PV product, so the load of K_{j+2} starts a whole tile earlier
  // than with a joint slot and the loads stay off the critical path.
  const uint32_t q_full = bar0;
  auto k_full = [&](int s) { return bar0 + 8u * (1 + s); };
  auto k_empty = [&](int s) { return bar0 + 8u * (3 + s); };
  auto v_full = [&](int s) { return bar0 + 8u * (5 + s); };
  auto v_empty = [&](int s) { return bar0 + 8u * (7 + s); };
  auto s_full = [&](int b) { return bar0 + 8u * (9 + b); };
  auto s_free = [&](int b) { return bar0 + 8u * (11 + b); };
  const uint32_t p_full = bar0 + 8u * 13, p_free = bar0 + 8u * 14;
  const uint32_t o_full = bar0 + 8u * 15;             // the last PV product has completed
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(smem + BAR_OFF - CUT + 24 * 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.y;
  const int hk = h / (p.nq / p.nkv);
  const int q_begin = p.cu_q[b], q_len = p.cu_q[b + 1] - q_begin;
  const int n_q_tiles = (q_len + kBM - 1) / kBM;
  if ((int)blockIdx.x >= n_q_tiles) return;          // uniform for the whole CTA: nothing allocated yet
  const int m0 = (n_q_tiles - 1 - (int)blockIdx.x) * kBM;  // heavy (late) tiles first
  const int kv_len = p.kv_lens[b];
  const int ctx_off = kv_len - q_len;                 // absolute position of this chunk's first query
  const int kv_hi = p.causal ? min(kv_len, ctx_off + m0 + kBM) : kv_len;
  const int first = p.window > 0 ? max(0, ctx_off + m0 - p.window + 1) / kBN : 0;   // tiles before every row's window
  const int kept = min((p.keep + kBN - 1) / kBN, first);                             // tiles of kept positions ahead of it
  const int n_tiles = kept + (kv_hi + kBN - 1) / kBN - first;
  const auto tile_of = [&](int j) { return j < kept ? j : j - kept + first; };

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(o_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(k_full(s), 1);
      mbar_init(k_empty(s), 1);
      mbar_init(v_full(s), 1);
      mbar_init(v_empty(s), 1);
      mbar_init(s_full(s), 1);
      mbar_init(s_free(s), 8);
    }
    mbar_init(p_full, 8);
    mbar_init(p_free, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_holder)), "r"(TMEM_COLS));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  const uint32_t TS0 = tmem, TO0 = tmem + 256;        // S[b] = TS0 + 128 b; O accumulates at TO0 over all tiles

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      mbar_expect_tx(q_full, kTile);
      tma_load_2d(sbase + Q_OFF, &tma_q, h * kD, q_begin + m0, q_full);
      tma_load_2d(sbase + Q_OFF + kHalf, &tma_q, h * kD + 64, q_begin + m0, q_full);
    }
    const int pages = kBN / p.page;                   // pages per kv tile (page is 16, 32, 64 or 128)
    const int32_t* bt = p.block_table + (int64_t)b * p.bt_stride;
    const int n_blk = (kv_len + p.page - 1) / p.page;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int st = j & 1;
      const int pg = tile_of(j) * pages + lane;
      const int myblk = (lane < pages && pg < n_blk) ? bt[pg] : 0;   // pages past the sequence read block 0 (masked)
      const int y = p.rows_kv ? myblk * p.page : (myblk * p.nkv + hk) * p.page;
      const int x = p.rows_kv ? hk * kD : 0;
      const uint32_t off = (uint32_t)(lane * p.page * 128);
      const uint32_t kdst = sbase + KV_OFF + st * KV_STAGE, vdst = kdst + kTile;
      // every lane gathers its own page: the copies of all pages issue together
      if (!mbar_wait_warp(k_empty(st), ((j >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
      if (lane == 0) mbar_expect_tx(k_full(st), kTile);
      __syncwarp();
      if (lane < pages) {
        tma_load_2d(kdst + off, &tma_k, x, y, k_full(st));
        tma_load_2d(kdst + kHalf + off, &tma_k, x + 64, y, k_full(st));
      }
      if constexpr (LSE) continue;
      if (!mbar_wait_warp(v_empty(st), ((j >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
      if (lane == 0) mbar_expect_tx(v_full(st), kTile);
      __syncwarp();
      if (lane < pages) {
        tma_load_2d(vdst + off, &tma_v, x, y, v_full(st));
        tma_load_2d(vdst + kHalf + off, &tma_v, x + 64, y, v_full(st));
      }
      __syncwarp();
    }
    if (!ok) {
      const long long t0 = clock64();
      while (clock64() - t0 < 20000000LL) {}          // bounded grace period for copies in flight
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    constexpr uint32_t ID_QK = idesc(false, 128), ID_PV = idesc(true, 128);
    bool ok = mbar_wait_warp(q_full, 0, abort_flag);
    auto issue_qk = [&](int j) {
      // S[j & 1] = Q K_j^T : 8 steps of 16 along head_dim, two 64-element halves
      const uint32_t kaddr = sbase + KV_OFF + (j & 1) * KV_STAGE;
      if (lane == 0) {
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          const uint32_t o = (ks >> 2) * kHalf + (ks & 3) * 32;
          umma(TS0 + (j & 1) * 128, smem_desc(sbase + Q_OFF + o, 16, 1024), smem_desc(kaddr + o, 16, 1024), ID_QK, ks != 0);
        }
        if constexpr (LSE) umma_commit(k_empty(j & 1));   // the last commit of all is one that somebody waits for
        umma_commit(s_full(j & 1));
        if constexpr (!LSE) umma_commit(k_empty(j & 1));  // the K slot may be refilled once these MMAs have read it
      }
      __syncwarp();
    };
    if (ok && n_tiles > 0) {
      ok = mbar_wait_warp(k_full(0), 0, abort_flag);
      tc_fence_after();
      if (ok) issue_qk(0);
    }
    for (int j = 0; j < n_tiles && ok; ++j) {
      if (j + 1 < n_tiles) {
        const int nb = (j + 1) & 1, use = (j + 1) >> 1;
        if (!mbar_wait_warp(k_full(nb), use & 1, abort_flag)) { ok = false; break; }
        if (!mbar_wait_warp(s_free(nb), (use & 1) ^ 1, abort_flag)) { ok = false; break; }
        tc_fence_after();
        issue_qk(j + 1);
      }
      if constexpr (LSE) continue;
      if (!mbar_wait_warp(v_full(j & 1), (j >> 1) & 1, abort_flag)) { ok = false; break; }
      if (!mbar_wait_warp(p_full, j & 1, abort_flag)) { ok = false; break; }   // also: O has been rescaled if need be
      tc_fence_after();
      if (lane == 0) {
        // O += P V_j : 8 steps of 16 kv tokens; V is MN-major (rows = tokens, 128-byte rows of
        // 64 head_dim elements, second half of head_dim one half-tile further)
        const uint32_t vaddr = sbase + KV_OFF + (j & 1) * 2 * kTile + kTile;
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          const uint32_t pa = sbase + P_OFF + (ks >> 2) * kHalf + (ks & 3) * 32;
          umma(TO0, smem_desc(pa, 16, 1024), smem_desc(vaddr + ks * 16 * 128, kHalf, 1024), ID_PV, (j | ks) != 0);
        }
        umma_commit(p_free);
        if (j == n_tiles - 1) umma_commit(o_full);
        umma_commit(v_empty(j & 1));
      }
      __syncwarp();
    }
  } else {
    // ------------------------------------------------------------------ softmax / output (warps 2..9)
    // Two threads per query row: warps 2-5 take kv columns / head_dim columns 0..63 of the row, warps
    // 6-9 take 64..127 (two warps per scheduler hide each other's TMEM round trips, and 64 instead of
    // 128 output values per thread leave room to keep the S row in registers: S is read once).
    const int quarter = warp & 3;                     // TMEM lanes this warp may read
    const int half = (warp - 2) >> 2;                 // which 64 columns
    const int row = quarter * 32 + lane;              // query row inside the tile
    const uint32_t lane_addr = (uint32_t)(quarter * 32) << 16;
    const int q_pos = ctx_off + m0 + row;             // absolute position of this query token
    const int limit = p.causal ? min(kv_len - 1, q_pos) : kv_len - 1;   // last kv index this row may see
    const int low = p.window > 0 ? q_pos - p.window + 1 : 0;            // the first one
    float* smax = reinterpret_cast<float*>(smem + XCH_OFF - CUT);             // [2 tile parities][2 halves][128 rows]
    float* lsum = smax + 2 * 2 * kBM;                                   // [2 halves][128 rows]
    // O stays in TMEM and the MMAs accumulate into it over all kv tiles.  The exponent uses a row
    // maximum m that lags the true one: it moves (and O and l are rescaled) only when the true
    // maximum has grown by more than 2^kLag, so after the first tiles the rescale is rare and the
    // common tile costs no pass over O at all.  P stays below 2^kLag, well inside bf16 and fp32 range.
    constexpr float kLag = 8.f;
    const float sc = CAP ? 1.f : p.scale_log2;        // capped scores are in the log2 domain already
    float m = -INFINITY, l = 0.f;
    if (p.sink != nullptr) {                          // a key with this score and no value
      m = p.sink[h] * 1.4426950408889634f;
      if (half == 0) l = 1.f;                         // the two halves of a row add their sums
    }
    bool ok = true;
    const uint32_t oaddr = TO0 + half * 64 + lane_addr;
    // Every thread runs every iteration and every named barrier even after a wait has given up (the
    // waits then fail at once): a thread that left early would strand its partners in bar.sync.
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j & 1;
      ok = ok && mbar_wait(s_full(sb), (j >> 1) & 1, abort_flag);
      tc_fence_after();
      const uint32_t saddr = TS0 + sb * 128 + half * 64 + lane_addr;
      const int kv0 = tile_of(j) * kBN + half * 64;
      const bool full_tile = kv0 + 63 <= limit && (kv0 >= low || kv0 + 63 < p.keep);
      uint32_t sv[64];
      tmem_ld32(saddr, sv);
      tmem_ld32(saddr + 32, sv + 32);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(s_free(sb));         // S has been read out: the next QK may overwrite it
      if constexpr (CAP) {
        float top = 0.f;
#pragma unroll
        for (int i = 0; i < 64; ++i) top = fmaxf(top, fabsf(__uint_as_float(sv[i])));
        if (__all_sync(0xffffffffu, top <= p.cap.small)) {
#pragma unroll
          for (int i = 0; i < 64; ++i) sv[i] = __float_as_uint(soft_cap_small(__uint_as_float(sv[i]), p.cap));
        } else {
#pragma unroll
          for (int i = 0; i < 64; ++i) sv[i] = __float_as_uint(soft_cap(__uint_as_float(sv[i]), p.cap));
        }
      }
      if (!full_tile) {                               // bit i: column i is seen
        const auto below = [&](int t) {               // columns of positions before t
          const int n = min(max(t - kv0, 0), 64);
          return n == 64 ? ~0ull : (1ull << n) - 1;
        };
        const unsigned long long seen = below(limit + 1) & (~below(low) | below(p.keep));
        const uint32_t s0 = (uint32_t)seen, s1 = (uint32_t)(seen >> 32);
#pragma unroll
        for (int i = 0; i < 64; ++i)
          if (!((i < 32 ? s0 : s1) & (1u << (i & 31)))) sv[i] = 0xff800000u;      // -inf
      }
      if constexpr (LSE && CAP) {
        if (p.cap.out <= 100.f) {                     // sums of 2^score stay within fp32 without a reference
          m = 0.f;
          float rs = 0.f;
#pragma unroll
          for (int i = 0; i < 64; ++i) rs += exp2f(__uint_as_float(sv[i]));
          l += rs;
          continue;
        }
      }
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < 64; ++i) mx = fmaxf(mx, __uint_as_float(sv[i]));
      smax[(sb * 2 + half) * kBM + row] = mx;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      mx = fmaxf(mx, smax[(sb * 2 + (half ^ 1)) * kBM + row]);
      const float m_true = fmaxf(m, mx * sc);
      float factor = 1.f;
      if (m_true - m > kLag) {                        // also the first tile that shows this row a key (m = -inf)
        factor = exp2f(m - m_true);                   // 0 when m was -inf: nothing accumulated yet
        m = m_true;
      }
      const float m_use = m == -INFINITY ? 0.f : m;
      if constexpr (LSE) {
        float rs = 0.f;
#pragma unroll
        for (int i = 0; i < 64; ++i) rs += exp2f(__uint_as_float(sv[i]) * sc - m_use);
        l = l * factor + rs;
        continue;
      }
      // P may be overwritten, and O touched, once the PV product of the previous tile has completed
      ok = ok && mbar_wait(p_free, (j & 1) ^ 1, abort_flag);
      if (j > 0 && __any_sync(0xffffffffu, factor != 1.f)) {
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          uint32_t r[32];
          tmem_ld32(oaddr + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * factor);
          tmem_st32(oaddr + c * 32, r);
        }
        tmem_st_wait();
        tc_fence_before();
      }
      float rs = 0.f;
      const uint32_t pbase = sbase + P_OFF + half * kHalf + row * 128;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        uint32_t packed[4];
#pragma unroll
        for (int e = 0; e < 8; e += 2) {
          const int i = u * 8 + e;
          const float p0 = exp2f(__uint_as_float(sv[i]) * sc - m_use);
          const float p1 = exp2f(__uint_as_float(sv[i + 1]) * sc - m_use);
          rs += p0 + p1;
          const __nv_bfloat162 pb = __floats2bfloat162_rn(p0, p1);
          packed[e >> 1] = *reinterpret_cast<const uint32_t*>(&pb);
        }
        const uint32_t dst = pbase + ((u ^ (row & 7)) << 4);
        asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(dst), "r"(packed[0]), "r"(packed[1]), "r"(packed[2]),
                     "r"(packed[3])
                     : "memory");
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
      l = l * factor + rs;
    }
    float o[64];
    if (!LSE && n_tiles > 0) {
      ok = ok && mbar_wait(o_full, 0, abort_flag);
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t r[32];
        tmem_ld32(oaddr + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = __uint_as_float(r[i]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < 64; ++i) o[i] = 0.f;
    }
    // ---- output: the two halves of a row add their sums, normalise, stage the tile in shared memory
    // (the Q buffer is free now), store rows
    lsum[half * kBM + row] = l;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    l += lsum[(half ^ 1) * kBM + row];
    const float inv = l > 0.f ? 1.f / l : 0.f;
    if (p.lse != nullptr && half == 0 && ok && m0 + row < q_len)
      p.lse[(int64_t)(q_begin + m0 + row) * p.nq + h] = l > 0.f ? m + log2f(l) : -INFINITY;
    uint8_t* stage = smem + Q_OFF;                    // [128 rows][256 bytes], 16-byte units XOR-swizzled by row
#pragma unroll
    for (int u = 0; u < (LSE ? 0 : 8); ++u) {
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = o[u * 8 + e] * inv;
      const bf16x8 v = pack8(f);
      *reinterpret_cast<uint4*>(stage + row * 256 + (((half * 8 + u) ^ (row & 15)) << 4)) = *reinterpret_cast<const uint4*>(&v);
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    if (!LSE && ok) {
      const int t = threadIdx.x - 64;                 // 0..255
      const int u = t & 15;
      for (int r0 = t >> 4; r0 < kBM; r0 += 16) {     // 16 rows per pass, 16 threads x 16 bytes per row
        if (m0 + r0 < q_len) {
          const uint4 v = *reinterpret_cast<const uint4*>(stage + r0 * 256 + ((u ^ (r0 & 15)) << 4));
          *reinterpret_cast<uint4*>(p.out + (int64_t)(q_begin + m0 + r0) * p.o_stride + h * kD + u * 8) = v;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && *abort_flag && p.err != nullptr) atomicExch(p.err, 1);
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(TMEM_COLS));
  }
}

// Weights that another kernel left in memory times the values: one CTA = (sequence, query head, tile of 128 rows of a window of
// batch rows), 192 threads, two CTAs an SM: warp 0 loads 64 keys of weights and gathers the values' pages (TMA, three stages), warp
// 1 issues the products into one TMEM accumulator, warps 2-5 store it.
struct WvParams {
  bf16* out;                   // [total_q, nq, dv]
  const int32_t *block_table, *cu_q, *kv_lens;
  int64_t w_rows;              // rows a head takes in the table of weights
  int dv, bt_stride, nq, nkv, page, row0, rows;
  int* err;
};
constexpr int kWvStages = 3, kWvKeys = 64;
constexpr int kWvW = kBM * kWvKeys * 2, kWvV = kWvKeys * kD * 2;     // bytes of a stage's weights and values
constexpr int WV_BAR = kWvStages * (kWvW + kWvV);
constexpr int WV_SMEM = WV_BAR + 64 + 16 + 1024;

__global__ void __launch_bounds__(192, 2)
weights_values_kernel(const __grid_constant__ CUtensorMap tma_w, const __grid_constant__ CUtensorMap tma_v, const WvParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem), bar0 = sbase + WV_BAR;
  auto full = [&](int s) { return bar0 + 8u * s; };
  auto empty = [&](int s) { return bar0 + 8u * (kWvStages + s); };
  const uint32_t o_full = bar0 + 8u * 2 * kWvStages;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(smem + WV_BAR + 64);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.y, hk = h / (p.nq / p.nkv);
  const int q_end = p.cu_q[b + 1], q_lo = max(p.cu_q[b], p.row0), q_hi = min(q_end, p.row0 + p.rows);
  const int n_q_tiles = q_hi > q_lo ? (q_hi - q_lo + kBM - 1) / kBM : 0;
  if ((int)blockIdx.x >= n_q_tiles) return;          // uniform for the whole CTA: nothing allocated yet
  const int r0 = q_lo + (n_q_tiles - 1 - (int)blockIdx.x) * kBM;   // heavy (late) tiles first
  const int kv_len = p.kv_lens[b];
  const int kv_hi = min(kv_len, kv_len - (q_end - r0) + kBM);
  const int n_tiles = max(0, (kv_hi + kWvKeys - 1) / kWvKeys);
  if (threadIdx.x == 0) {
    for (int s = 0; s < kWvStages; ++s) {
      mbar_init(full(s), 1);
      mbar_init(empty(s), 1);
    }
    mbar_init(o_full, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_holder)), "r"(128));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  if (warp == 0) {
    const int per = min(p.page, kWvKeys), copies = kWvKeys / per;      // tokens of a copy
    const int32_t* bt = p.block_table + (int64_t)b * p.bt_stride;
    const int wy = (int)(h * p.w_rows) + r0 - p.row0;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int st = j % kWvStages, tok = j * kWvKeys + lane * per;
      const int blk = lane < copies && tok < kv_len ? bt[tok / p.page] : 0;            // past the sequence: block 0, weights 0
      const int y = (blk * p.nkv + hk) * p.page + tok % p.page;
      const uint32_t wdst = sbase + st * (kWvW + kWvV), vdst = wdst + kWvW, off = (uint32_t)(lane * per * 128);
      if (!mbar_wait_warp(empty(st), ((j / kWvStages) & 1) ^ 1, abort_flag)) { ok = false; break; }
      if (lane == 0) {
        mbar_expect_tx(full(st), kWvW + kWvV);
        tma_load_2d(wdst, &tma_w, j * kWvKeys, wy, full(st));
      }
      __syncwarp();
      if (lane < copies) {
        tma_load_2d(vdst + off, &tma_v, 0, y, full(st));
        tma_load_2d(vdst + kWvV / 2 + off, &tma_v, 64, y, full(st));
      }
      __syncwarp();
    }
    if (!ok) {
      const long long t0 = clock64();
      while (clock64() - t0 < 20000000LL) {}          // bounded grace period for copies in flight
    }
  } else if (warp == 1) {
    constexpr uint32_t ID_PV = idesc(true, 128);
    for (int j = 0; j < n_tiles; ++j) {
      const int st = j % kWvStages;
      if (!mbar_wait_warp(full(st), (j / kWvStages) & 1, abort_flag)) break;
      tc_fence_after();
      if (lane == 0) {
        const uint32_t wa = sbase + st * (kWvW + kWvV), va = wa + kWvW;
#pragma unroll
        for (int ks = 0; ks < kWvKeys / 16; ++ks)
          umma(tmem, smem_desc(wa + ks * 32, 16, 1024), smem_desc(va + ks * 16 * 128, kWvV / 2, 1024), ID_PV, (j | ks) != 0);
        umma_commit(empty(st));
        if (j == n_tiles - 1) umma_commit(o_full);
      }
      __syncwarp();
    }
  } else {
    const int quarter = warp & 3, row = quarter * 32 + lane;
    bool ok = true;
    if (n_tiles > 0) {
      ok = mbar_wait_warp(o_full, 0, abort_flag);
      tc_fence_after();
    }
    bf16* dst = p.out + ((int64_t)(r0 + row) * p.nq + h) * p.dv;
    const bool live = ok && r0 + row < q_hi, vec = p.dv % 8 == 0;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      uint32_t r[32];
      if (n_tiles > 0) {
        tmem_ld32(tmem + ((uint32_t)(quarter * 32) << 16) + c * 32, r);
        tmem_ld_wait();
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = 0;
      }
      if (!live) continue;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int e = c * 32 + u * 8;
        float f[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(r[u * 8 + i]);
        if (vec) {
          if (e < p.dv) *reinterpret_cast<bf16x8*>(dst + e) = pack8(f);
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i)
            if (e + i < p.dv) dst[e + i] = __float2bfloat16(f[i]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && *abort_flag && p.err != nullptr) atomicExch(p.err, 1);
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(128));
  }
}

static int* g_err[64] = {};

}  // namespace fmha
}  // namespace xllm

// Same contract as xllm_paged_prefill_attn for head_dim 128, page_size in
// {16, 32, 64, 128}: q [total_q, nq, 128] (row stride q_stride elements), caches
// [n_blocks, nkv, page, 128], cu_q absolute row offsets [batch + 1], kv_lens [batch].
// `lse` (optional, fp32 [total_q, nq]) receives every row's log-sum-exp in the log2 domain, so that the
// result can be merged with attention over other keys (xllm_attn_merge, the beam-tail kernel).
static int prefill_tc(void* out, int64_t o_stride, const void* q, int64_t q_stride, int64_t total_q, const void* k_cache,
                      const void* v_cache, int64_t n_blocks, int64_t kv_ld, const void* block_table, int bt_stride,
                      const void* cu_q, const void* kv_lens, int batch, int max_q_len, int nq, int nkv, int page_size,
                      float scale, int causal, int window, int keep, float softcap, const void* sink, void* lse, void* stream) {
  using namespace xllm;
  using namespace xllm::fmha;
  if (batch == 0 || max_q_len == 0) return 0;
  if (nq % nkv != 0 || (page_size != 16 && page_size != 32 && page_size != 64 && page_size != 128) || q_stride % 8 ||
      o_stride % 8 || keep < 0 || kv_ld % 8 || (((uintptr_t)q | (uintptr_t)out | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15))
    return (int)cudaErrorInvalidValue;
  int dev = 0;
  cudaGetDevice(&dev);
  static bool attr_done[64] = {};
  if (!attr_done[dev & 63]) {
    cudaError_t e = cudaSuccess;
    for (const auto kernel : {prefill_tc_kernel<false, false>, prefill_tc_kernel<true, false>, prefill_tc_kernel<false, true>,
                              prefill_tc_kernel<true, true>})
      if (e == cudaSuccess) e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_TOTAL);
    if (e != cudaSuccess) return (int)e;
    attr_done[dev & 63] = true;
  }
  if (g_err[dev & 63] == nullptr) {
    if (cudaMalloc(&g_err[dev & 63], sizeof(int)) != cudaSuccess) return (int)cudaErrorMemoryAllocation;
    cudaMemset(g_err[dev & 63], 0, sizeof(int));
  }
  CUtensorMap tq, tk, tv;
  const int64_t cache_rows = kv_ld > 0 ? n_blocks * page_size : n_blocks * nkv * page_size;
  const int64_t cols = kv_ld > 0 ? (int64_t)nkv * kD : kD, ld = kv_ld > 0 ? kv_ld : kD;
  if (!make_map(&tq, q, total_q, (int64_t)nq * kD, q_stride, kBM) || !make_map(&tk, k_cache, cache_rows, cols, ld, page_size) ||
      !make_map(&tv, v_cache, cache_rows, cols, ld, page_size))
    return (int)cudaErrorInvalidValue;
  Params p;
  p.out = (bf16*)out; p.block_table = (const int32_t*)block_table; p.cu_q = (const int32_t*)cu_q;
  p.kv_lens = (const int32_t*)kv_lens; p.o_stride = o_stride; p.bt_stride = bt_stride; p.nq = nq; p.nkv = nkv;
  p.page = page_size; p.causal = causal; p.window = window; p.scale_log2 = scale * 1.4426950408889634f; p.err = g_err[dev & 63];
  p.lse = (float*)lse; p.sink = (const float*)sink; p.keep = window > 0 ? keep : 0; p.rows_kv = kv_ld > 0; p.cap = make_soft_cap(scale, softcap);
  dim3 grid((max_q_len + kBM - 1) / kBM, nq, batch);
  const auto kernel = out == nullptr ? (softcap > 0.f ? prefill_tc_kernel<true, true> : prefill_tc_kernel<false, true>)
                                     : (softcap > 0.f ? prefill_tc_kernel<true, false> : prefill_tc_kernel<false, false>);
  kernel<<<grid, 320, out == nullptr ? SMEM_TOTAL - LSE_CUT : SMEM_TOTAL, (cudaStream_t)stream>>>(tq, tk, tv, p);
  return XLLM_LAUNCH_CHECK();
}

XLLM_API int xllm_paged_prefill_attn_tc_lse(void* out, int64_t o_stride, const void* q, int64_t q_stride, int64_t total_q,
                                            const void* k_cache, const void* v_cache, int64_t n_blocks,
                                            const void* block_table, int bt_stride, const void* cu_q,
                                            const void* kv_lens, int batch, int max_q_len, int nq, int nkv,
                                            int page_size, float scale, int causal, int window, void* lse, void* stream) {
  return prefill_tc(out, o_stride, q, q_stride, total_q, k_cache, v_cache, n_blocks, 0, block_table, bt_stride, cu_q, kv_lens,
                    batch, max_q_len, nq, nkv, page_size, scale, causal, window, 0, 0.f, nullptr, lse, stream);
}

// The same with kept first positions beside the window, soft-capped scores and sinks (see xllm_paged_prefill_attn_kept).
// kv_ld > 0: K and V are matrices [n_blocks * page_size, nkv * 128] of that row stride, a page being page_size rows.
XLLM_API int xllm_paged_prefill_attn_tc_kept(void* out, int64_t o_stride, const void* q, int64_t q_stride, int64_t total_q,
                                             const void* k_cache, const void* v_cache, int64_t n_blocks, int64_t kv_ld,
                                             const void* block_table, int bt_stride, const void* cu_q, const void* kv_lens,
                                             int batch, int max_q_len, int nq, int nkv, int page_size, float scale, int causal,
                                             int window, int keep, float softcap, const void* sink, void* stream) {
  return prefill_tc(out, o_stride, q, q_stride, total_q, k_cache, v_cache, n_blocks, kv_ld, block_table, bt_stride, cu_q,
                    kv_lens, batch, max_q_len, nq, nkv, page_size, scale, causal, window, keep, softcap, sink, nullptr, stream);
}

XLLM_API int xllm_paged_prefill_attn_tc(void* out, int64_t o_stride, const void* q, int64_t q_stride, int64_t total_q,
                                        const void* k_cache, const void* v_cache, int64_t n_blocks,
                                        const void* block_table, int bt_stride, const void* cu_q, const void* kv_lens,
                                        int batch, int max_q_len, int nq, int nkv, int page_size, float scale,
                                        int causal, int window, void* stream) {
  return xllm_paged_prefill_attn_tc_lse(out, o_stride, q, q_stride, total_q, k_cache, v_cache, n_blocks, block_table,
                                        bt_stride, cu_q, kv_lens, batch, max_q_len, nq, nkv, page_size, scale, causal,
                                        window, nullptr, stream);
}

// lse [total_q, nq] fp32: the log-sum-exp (log2 domain) of every row's scores over all it may see, and nothing else.
XLLM_API int xllm_prefill_lse_tc(void* lse, const void* q, int64_t q_stride, int64_t total_q, const void* k_cache, int64_t n_blocks,
                                 const void* block_table, int bt_stride, const void* cu_q, const void* kv_lens, int batch,
                                 int max_q_len, int nq, int nkv, int page_size, float scale, float softcap, void* stream) {
  if (lse == nullptr) return (int)cudaErrorInvalidValue;
  return prefill_tc(nullptr, 0, q, q_stride, total_q, k_cache, k_cache, n_blocks, 0, block_table, bt_stride, cu_q, kv_lens, batch,
                    max_q_len, nq, nkv, page_size, scale, 1, 0, 0, softcap, nullptr, lse, stream);
}

// Rows [row0, row0 + rows) of out [total_q, nq, dv] = tables of weights times the values of each head's key/value head:
// w [nq, w_rows, ld] bf16, row r - row0 of head h; a row's weights are defined (zero beyond what it sees) up to the last key that
// its tile of 128 rows sees, rounded up to 128.  v_cache [n_blocks, nkv, page, 128]; ld a multiple of 128.
XLLM_API int xllm_talk_values_tc(void* out, int dv, const void* w, int64_t w_rows, int64_t ld, const void* v_cache, int64_t n_blocks,
                                 const void* block_table, int bt_stride, const void* cu_q, const void* kv_lens, int batch,
                                 int max_q_len, int row0, int rows, int nq, int nkv, int page_size, void* stream) {
  using namespace xllm;
  using namespace xllm::fmha;
  if (batch == 0 || rows == 0 || max_q_len == 0) return 0;
  if (nq % nkv != 0 || (page_size != 16 && page_size != 32 && page_size != 64 && page_size != 128) || ld <= 0 || ld % 128 || dv <= 0 ||
      dv > kD || w_rows < rows || (((uintptr_t)w | (uintptr_t)v_cache) & 15))
    return (int)cudaErrorInvalidValue;
  int dev = 0;
  cudaGetDevice(&dev);
  static bool attr_done[64] = {};
  if (!attr_done[dev & 63]) {
    const cudaError_t e = cudaFuncSetAttribute(weights_values_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, WV_SMEM);
    if (e != cudaSuccess) return (int)e;
    attr_done[dev & 63] = true;
  }
  if (g_err[dev & 63] == nullptr) {
    if (cudaMalloc(&g_err[dev & 63], sizeof(int)) != cudaSuccess) return (int)cudaErrorMemoryAllocation;
    cudaMemset(g_err[dev & 63], 0, sizeof(int));
  }
  CUtensorMap tw, tv;
  if (!make_map(&tw, w, (int64_t)nq * w_rows, ld, ld, kBM) || !make_map(&tv, v_cache, n_blocks * nkv * page_size, kD, kD, min(page_size, kWvKeys)))
    return (int)cudaErrorInvalidValue;
  WvParams p{(bf16*)out, (const int32_t*)block_table, (const int32_t*)cu_q, (const int32_t*)kv_lens, w_rows, dv, bt_stride, nq, nkv,
             page_size, row0, rows, g_err[dev & 63]};
  const dim3 grid((min(max_q_len, rows) + kBM - 1) / kBM, nq, batch);
  weights_values_kernel<<<grid, 192, WV_SMEM, (cudaStream_t)stream>>>(tw, tv, p);
  return XLLM_LAUNCH_CHECK();
}

// 0 = no bounded wait expired in the prefill kernel on this device since the last call.
XLLM_API int xllm_fmha_error_status() {
  using namespace xllm::fmha;
  int dev = 0;
  cudaGetDevice(&dev);
  if (g_err[dev & 63] == nullptr) return 0;
  int v = 0;
  cudaMemcpy(&v, g_err[dev & 63], sizeof(int), cudaMemcpyDeviceToHost);
  if (v != 0) cudaMemset(g_err[dev & 63], 0, sizeof(int));
  return v;
}
