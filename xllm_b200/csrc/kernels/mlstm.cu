// Matrix memory with exponential gates and a running maximum (mLSTM of xLSTM), per head:
//
//   i = cap tanh(zi / cap);   f = logsigmoid(cap tanh(zf / cap));   m' = max(f + m, i)
//   S <- exp(f + m - m') S + exp(i - m') k v^T;   n <- exp(f + m - m') n + exp(i - m') k
//   o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)                    S [dk, dv], n [dk], m: fp32, one of each per state slot
//
// m starts at 0.  zi and zf are fp32 projections; q is scaled.  The output of a head is divided by its root mean square,
// weighted (a weight for every head's element) and multiplied by the sigmoid of a gate.
//
//   mlstm_decode_kernel     one token per sequence, from the projection rows to the finished row; the state crosses HBM
//                           once in each direction
//   mlstm_gates_kernel,     prompts, bf16: sixteen tokens at a time on the tensor cores.  A scan over (sum of f, maximum)
//   mlstm_chunk_kernel      gives every token's m; with F the sum of f since the chunk's start, token t sees token s of its
//                           chunk with weight exp(F_t - F_s + i_s - m_t) and the state before the chunk with
//                           exp(F_t + m_before - m_t), all of them at most 1.  A warp owns 16 state columns for all of dk
//                           as fp32 accumulators of S^T, which are the A operand of O^T = S^T Q^T without leaving the
//                           registers; so are the token-token weights (B operand of V^T P^T).  q, k and v are bf16 as
//                           projected; S, the weights and the weighted v enter the products as a sum of two bf16 terms
//   mlstm_prefill_kernel    prompts of any type and size: token by token in fp32 with the state in registers
//                           (recurrence.cuh)
// One more warp keeps n, as the state column of a value that is always 1.  Raw sums and denominators go to head_norm.cu.
//
// A sequence whose rows in the batch are its first tokens (kv_len == number of rows) starts from zero whatever its slot
// holds; slot < 0 marks padding rows.  Built without fast-math: errors of the gates multiply up over a sequence.
#include "attn_common.cuh"
#include "recurrence.cuh"
#include "short_conv.cuh"

namespace xllm {

template <typename T>
struct MlstmParams {
  float *state, *norm, *top;     // [slots, H, dk, dvp], [slots, H, dk], [slots, H]
  const int32_t *slots, *cu_q, *kv_lens;
  const T *q, *k, *v;            // column blocks of the projection rows
  int64_t ld;
  const float *zi, *zf;          // [rows, z_ld]: head h in column h
  int64_t z_ld;
  const T* gate;                 // [rows, gate_ld] (decode)
  int64_t gate_ld;
  const T* norm_w;               // [H dv]
  T* out;                        // [rows, out_ld] (decode)
  int64_t out_ld;
  float *o, *div;                // [rows, H, dv], [rows, H] (prompts)
  int H, dk, dv, dvp;
  float q_scale, cap, eps;
};

__device__ __forceinline__ float log_sigmoid_exact(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

constexpr float kDivEps = 1e-6f;

// ------------------------------------------------------------------------------------------------ decode
// grid (heads, sequences), 256 threads: dvp / 4 column groups x row groups, NR rows of four columns per thread.
template <typename T, int NR>
__global__ void __launch_bounds__(256, NR <= 8 ? 3 : (NR <= 16 ? 2 : 1)) mlstm_decode_kernel(MlstmParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  const int dk = p.dk, dv = p.dv, dvp = p.dvp, dkp = (dk + 3) & ~3;
  float* qs = sm;
  float* ks = qs + dkp;
  float* vs = ks + dkp;                    // [dvp]
  float* red = vs + dvp;                   // [RG][dvp]
  __shared__ float red32[32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int CG = dvp >> 2, RG = 256 / CG;
  const int cg = tid % CG, rg = tid / CG;
  pdl_wait();
  pdl_launch_dependents();
  T* orow = p.out + b * p.out_ld + (int64_t)h * dv;
  const int slot = p.slots[b], len = p.kv_lens[b];
  if (slot < 0 || len <= 0) {
    for (int i = tid; i < dv; i += 256) orow[i] = from_f32<T>(0.f);
    return;
  }
  const bool active = rg < RG, fresh = len == 1;
  const int64_t sh = (int64_t)slot * p.H + h;
  float* S = p.state + sh * dk * dvp + cg * 4;
  float4 s[NR];
#pragma unroll
  for (int u = 0; u < NR; ++u) {
    const int r = rg + u * RG;
    s[u] = (active && !fresh && r < dk) ? *reinterpret_cast<const float4*>(S + (int64_t)r * dvp)
                                        : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float i_log = p.cap * tanhf(p.zi[b * p.z_ld + h] / p.cap);
  const float f_log = log_sigmoid_exact(p.cap * tanhf(p.zf[b * p.z_ld + h] / p.cap));
  const float m_old = fresh ? 0.f : p.top[sh];
  const float m = fmaxf(f_log + m_old, i_log);
  const float keep = expf(f_log + m_old - m), write = expf(i_log - m);
  const T* qr = p.q + b * p.ld + (int64_t)h * dk;
  const T* kr = p.k + b * p.ld + (int64_t)h * dk;
  const T* vr = p.v + b * p.ld + (int64_t)h * dv;
  float nq = 0.f;
  for (int i = tid; i < dk; i += 256) {
    const float qq = to_f32(qr[i]) * p.q_scale, kk = to_f32(kr[i]) * write;
    qs[i] = qq;
    ks[i] = kk;
    const float n = (fresh ? 0.f : keep * p.norm[sh * dk + i]) + kk;
    p.norm[sh * dk + i] = n;
    nq += n * qq;
  }
  for (int i = tid; i < dvp; i += 256) vs[i] = i < dv ? to_f32(vr[i]) : 0.f;
  nq = block_sum(nq, red32);               // also the barrier behind qs, ks, vs and the reads of top
  if (tid == 0) p.top[sh] = m;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    const float4 v4 = *reinterpret_cast<const float4*>(vs + cg * 4);
#pragma unroll
    for (int u = 0; u < NR; ++u) {
      const int r = rg + u * RG;
      if (r >= dk) break;
      const float kk = ks[r], qq = qs[r];
      float4 x = s[u];
      x.x = keep * x.x + kk * v4.x; x.y = keep * x.y + kk * v4.y; x.z = keep * x.z + kk * v4.z; x.w = keep * x.w + kk * v4.w;
      *reinterpret_cast<float4*>(S + (int64_t)r * dvp) = x;
      o.x += qq * x.x; o.y += qq * x.y; o.z += qq * x.z; o.w += qq * x.w;
    }
    *reinterpret_cast<float4*>(red + rg * dvp + cg * 4) = o;
  }
  __syncthreads();
  float mine = 0.f, ss = 0.f;              // dv <= 128: one element per thread
  if (tid < dv) {
    for (int w = 0; w < RG; ++w) mine += red[w * dvp + tid];
    mine /= fmaxf(fabsf(nq), expf(-m)) + kDivEps;
    ss = mine * mine;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red32) / (float)dv + p.eps);
  if (tid < dv)
    orow[tid] = from_f32<T>(mine * inv * to_f32(p.norm_w[(int64_t)h * dv + tid]) *
                            sigmoid_as<T>(to_f32(p.gate[b * p.gate_ld + (int64_t)h * dv + tid])));
}

// ------------------------------------------------------------------------------------------------ prompts
// grid (column slices, heads, sequences); `warps` warps of eight columns and one more that keeps n (first slice only).
// V: elements fetched together (4 needs aligned rows).  Tiles are fetched into registers one tile ahead and converted on
// their way to shared memory; k takes its input gate there.
constexpr int kMlstmWarps = 8;

template <typename T, int V>
struct RawVec;
template <>
struct RawVec<bf16, 4> { uint2 x; };
template <>
struct RawVec<float, 4> { float4 x; };
template <>
struct RawVec<bf16, 1> { bf16 x; };
template <>
struct RawVec<float, 1> { float x; };

template <typename T, int V, int J>
__global__ void __launch_bounds__(32 * (kMlstmWarps + 1)) mlstm_prefill_kernel(MlstmParams<T> p) {
  constexpr int DK = 32 * J, TT = kRecTile, COLS = kMlstmWarps * kRecCols, NT = 32 * (kMlstmWarps + 1);
  constexpr int UNROLL = J > 8 ? 1 : 2;
  constexpr int CK = DK / V, CV = COLS / V;                      // vectors per row
  constexpr int PER = (TT * (2 * CK + CV) + NT - 1) / NT;        // vectors per thread
  constexpr bool AHEAD = V == 4 && J <= 8;
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                                                // [TT][DK]
  float* ks = qs + TT * DK;
  float* vs = ks + TT * DK;                                      // [TT][COLS]
  __shared__ float keep_s[TT], write_s[TT], top_s[TT];
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool keeper = warp == kMlstmWarps;                       // the warp of n
  const int rgrp = lane & 7, c0 = blockIdx.x * COLS, lc = warp * kRecCols + (lane >> 3) * 2, col = c0 + lc;
  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q[b], n = p.cu_q[b + 1] - row0, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;
  const bool fresh = p.kv_lens[b] == n;
  const int64_t sh = (int64_t)slot * p.H + h;
  const bool live = keeper ? (blockIdx.x == 0 && lane < 8) : col < p.dvp;
  float* S = p.state + sh * p.dk * p.dvp + col;
  float* N = p.norm + sh * p.dk;
  StateColumns<J> st;
  if (!keeper) {
    st.load(S, p.dk, p.dvp, rgrp, live && !fresh);
  } else {
#pragma unroll
    for (int j = 0; j < J; ++j)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int r = 4 * (rgrp + 8 * j) + e;
        st.s[0][2 * j + e / 2] = pack_f2((live && !fresh && r < p.dk) ? N[r] : 0.f, (live && !fresh && r + 1 < p.dk) ? N[r + 1] : 0.f);
        st.s[1][2 * j + e / 2] = 0;
      }
  }
  float m_run = fresh ? 0.f : p.top[sh];                         // of the last token, kept by warp 0

  RawVec<T, V> ahead[AHEAD ? PER : 1];
  float zi = 0.f, zf = 0.f;
  // vector i of a tile: q rows, k rows, v rows
  const auto source = [&](int i, int t0, const T*& src, float*& dst, int& t, int& kind) {
    kind = i < TT * CK ? 0 : (i < 2 * TT * CK ? 1 : 2);
    const int w = kind == 2 ? CV : CK, at = i - kind * TT * CK;
    t = at / w;
    const int c = (at - t * w) * V;
    const int64_t row = row0 + t0 + t;
    bool ok = t0 + t < n && i < TT * (2 * CK + CV);
    if (kind == 2) {
      ok = ok && c0 + c < p.dv;
      src = p.v + row * p.ld + (int64_t)h * p.dv + c0 + c;
      dst = vs + t * COLS + c;
    } else {
      ok = ok && c < p.dk;
      src = (kind == 0 ? p.q : p.k) + row * p.ld + (int64_t)h * p.dk + c;
      dst = (kind == 0 ? qs : ks) + t * DK + c;
    }
    return ok;
  };
  const auto fetch = [&](int t0) {
    if constexpr (AHEAD) {
#pragma unroll
      for (int u = 0; u < PER; ++u) {
        const T* src;
        float* dst;
        int t, kind;
        if (source(tid + u * NT, t0, src, dst, t, kind)) ahead[u] = *reinterpret_cast<const RawVec<T, V>*>(src);
      }
    }
    if (warp == 0 && lane < TT && t0 + lane < n) {
      zi = p.zi[(int64_t)(row0 + t0 + lane) * p.z_ld + h];
      zf = p.zf[(int64_t)(row0 + t0 + lane) * p.z_ld + h];
    }
  };
  for (int i = tid; i < TT * (2 * DK + COLS); i += NT) sm[i] = 0.f;   // what lies behind dk and dv stays zero
  fetch(0);
  for (int t0 = 0; t0 < n; t0 += TT) {
    const int m = min(TT, n - t0);
    __syncthreads();                                             // the tile before is done with
    if (warp == 0) {
      // running maximum of the tile: token t maps m to max(a + m, c), and such maps compose
      float a = 0.f, c = -INFINITY, i_log = 0.f, f_log = 0.f;
      if (lane < m) {
        i_log = p.cap * tanhf(zi / p.cap);
        f_log = log_sigmoid_exact(p.cap * tanhf(zf / p.cap));
        a = f_log;
        c = i_log;
      }
#pragma unroll
      for (int d = 1; d < TT; d <<= 1) {
        const float pa = __shfl_up_sync(0xffffffffu, a, d), pc = __shfl_up_sync(0xffffffffu, c, d);
        if (lane >= d) {
          c = fmaxf(a + pc, c);
          a += pa;
        }
      }
      const float top = fmaxf(a + m_run, c);
      float prev = __shfl_up_sync(0xffffffffu, top, 1);
      if (lane == 0) prev = m_run;
      if (lane < m) {
        keep_s[lane] = expf(f_log + prev - top);
        write_s[lane] = expf(i_log - top);
        top_s[lane] = expf(-top);
      }
      m_run = __shfl_sync(0xffffffffu, top, m - 1);
    }
    __syncthreads();
    if constexpr (AHEAD) {
#pragma unroll
      for (int u = 0; u < PER; ++u) {
        const T* src;
        float* dst;
        int t, kind;
        if (source(tid + u * NT, t0, src, dst, t, kind)) {
          float x[V];
          load_f32<V>(reinterpret_cast<const T*>(&ahead[u]), x);
          const float f = kind == 0 ? p.q_scale : (kind == 1 ? write_s[t] : 1.f);
#pragma unroll
          for (int j = 0; j < V; ++j) x[j] *= f;
          store_f32<V>(dst, x);
        }
      }
    } else {
      for (int i = tid; i < TT * (2 * CK + CV); i += NT) {
        const T* src;
        float* dst;
        int t, kind;
        if (source(i, t0, src, dst, t, kind)) {
          float x[V];
          load_f32<V>(src, x);
          const float f = kind == 0 ? p.q_scale : (kind == 1 ? write_s[t] : 1.f);
#pragma unroll
          for (int j = 0; j < V; ++j) x[j] *= f;
          store_f32<V>(dst, x);
        }
      }
    }
    __syncthreads();
    if (t0 + TT < n) fetch(t0 + TT);
    if (keeper ? blockIdx.x != 0 : c0 + warp * kRecCols >= p.dv) continue;     // a warp without columns
    const float* vb = vs + lc;
    float* orow = p.o + ((int64_t)(row0 + t0) * p.H + h) * p.dv + col + (lane & 1);
    const bool writes = !keeper && rgrp < 2 && col + (lane & 1) < p.dv;
#pragma unroll UNROLL
    for (int t = 0; t < m; ++t) {
      f2 kf[2 * J], qf[2 * J];
      load_rows<J>(ks + t * DK, rgrp, kf);
      load_rows<J>(qs + t * DK, rgrp, qf);
      const float f = keep_s[t];
      const float2 v = keeper ? make_float2(1.f, 0.f) : *reinterpret_cast<const float2*>(vb + t * COLS);
      const f2 f_ = pack_f2(f, f), v0 = pack_f2(v.x, v.x), v1 = pack_f2(v.y, v.y);
      f2 d0 = 0, d1 = 0, e0 = 0, e1 = 0;                          // packed zeros
#pragma unroll
      for (int j = 0; j < 2 * J; j += 2) {
        st.s[0][j] = fma_f2(kf[j], v0, mul_f2(st.s[0][j], f_));
        st.s[1][j] = fma_f2(kf[j], v1, mul_f2(st.s[1][j], f_));
        st.s[0][j + 1] = fma_f2(kf[j + 1], v0, mul_f2(st.s[0][j + 1], f_));
        st.s[1][j + 1] = fma_f2(kf[j + 1], v1, mul_f2(st.s[1][j + 1], f_));
        d0 = fma_f2(st.s[0][j], qf[j], d0);
        d1 = fma_f2(st.s[1][j], qf[j], d1);
        e0 = fma_f2(st.s[0][j + 1], qf[j + 1], e0);
        e1 = fma_f2(st.s[1][j + 1], qf[j + 1], e1);
      }
      const float2 y0 = unpack_f2(add_f2(d0, e0)), y1 = unpack_f2(add_f2(d1, e1));
      const float y = sum_row_groups_2(y0.x + y0.y, y1.x + y1.y);
      if (writes) orow[(int64_t)t * p.H * p.dv] = y;
      if (keeper && lane == 0) p.div[(int64_t)(row0 + t0 + t) * p.H + h] = fmaxf(fabsf(y), top_s[t]) + kDivEps;
    }
  }
  if (!keeper) {
    if (live) st.store(S, p.dk, p.dvp, rgrp);
  } else if (live) {
#pragma unroll
    for (int j = 0; j < J; ++j)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int r = 4 * (rgrp + 8 * j) + e;
        const float2 a = unpack_f2(st.s[0][2 * j + e / 2]);
        if (r < p.dk) N[r] = a.x;
        if (r + 1 < p.dk) N[r + 1] = a.y;
      }
  }
}

// The running maximum behind the prompts, in a launch of its own: every slice of a head reads the one before them.
template <typename T>
__global__ void __launch_bounds__(256) mlstm_top_kernel(MlstmParams<T> p) {
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  __shared__ float wa[8], wc[8];
  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q[b], n = p.cu_q[b + 1] - row0, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;
  float* top = p.top + (int64_t)slot * p.H + h;
  float m = p.kv_lens[b] == n ? 0.f : *top;
  for (int t0 = 0; t0 < n; t0 += 256) {
    const int t = t0 + threadIdx.x;
    float a = 0.f, c = -INFINITY;
    if (t < n) {
      c = p.cap * tanhf(p.zi[(int64_t)(row0 + t) * p.z_ld + h] / p.cap);
      a = log_sigmoid_exact(p.cap * tanhf(p.zf[(int64_t)(row0 + t) * p.z_ld + h] / p.cap));
    }
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, a, d), pc = __shfl_up_sync(0xffffffffu, c, d);
      if (lane >= d) {
        c = fmaxf(a + pc, c);
        a += pa;
      }
    }
    if (lane == 31) { wa[warp] = a; wc[warp] = c; }
    __syncthreads();
    for (int w = 0; w < 8; ++w) m = fmaxf(wa[w] + m, wc[w]);
    __syncthreads();
  }
  if (threadIdx.x == 0) *top = m;
}

// ------------------------------------------------------------------------------------------------ prompts, chunks of 16
constexpr int kMC = 16;              // tokens per chunk
constexpr int kMStages = 4;
constexpr int kMWarps = 4;           // warps of 16 columns; one more for n

struct MlstmGates {
  float *a, *b, *em;                 // [H, rows]: i - F, F - m, exp(-m)
  float* before;                     // [H, chunks]: m before the chunk; chunk j of sequence s at cu_q[s] / 16 + s + j
  int rows, chunks;
};

// grid (heads, sequences), 256 threads; also leaves the running maximum behind the prompt in `top`
__global__ void __launch_bounds__(256) mlstm_gates_kernel(MlstmParams<bf16> p, MlstmGates g) {
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  __shared__ float wa[8], wc[8], wm[8];
  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q[b], n = p.cu_q[b + 1] - row0, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;
  float* top = p.top + (int64_t)slot * p.H + h;
  float m_in = p.kv_lens[b] == n ? 0.f : *top;
  const int64_t at = (int64_t)h * g.rows + row0;
  for (int t0 = 0; t0 < n; t0 += 256) {
    const int t = t0 + threadIdx.x;
    float f = 0.f, i = -INFINITY;
    if (t < n) {
      i = p.cap * tanhf(p.zi[(int64_t)(row0 + t) * p.z_ld + h] / p.cap);
      f = log_sigmoid_exact(p.cap * tanhf(p.zf[(int64_t)(row0 + t) * p.z_ld + h] / p.cap));
    }
    float F = f;                                     // within the chunk
#pragma unroll
    for (int d = 1; d < kMC; d <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, F, d, kMC);
      if ((lane & (kMC - 1)) >= d) F += up;
    }
    float a = f, c = i;                              // token maps m to max(a + m, c)
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, a, d), pc = __shfl_up_sync(0xffffffffu, c, d);
      if (lane >= d) {
        c = fmaxf(a + pc, c);
        a += pa;
      }
    }
    if (lane == 31) { wa[warp] = a; wc[warp] = c; }
    __syncthreads();
    float m_warp = m_in;                             // before this warp's tokens
    for (int w = 0; w < warp; ++w) m_warp = fmaxf(wa[w] + m_warp, wc[w]);
    const float m = fmaxf(a + m_warp, c);
    float prev = __shfl_up_sync(0xffffffffu, m, 1);
    if (lane == 0) prev = m_warp;
    if (t < n) {
      g.a[at + t] = i - F;
      g.b[at + t] = F - m;
      g.em[at + t] = expf(-m);
      if (t % kMC == 0) g.before[(int64_t)h * g.chunks + row0 / kMC + b + t / kMC] = prev;
    }
    for (int w = warp; w < 8; ++w) m_warp = fmaxf(wa[w] + m_warp, wc[w]);
    m_in = m_warp;
    __syncthreads();
  }
  if (threadIdx.x == 0) *top = m_in;
}

// grid (slices of 64 columns, heads, sequences)
template <int DK>
__global__ void __launch_bounds__(32 * (kMWarps + 1), DK > 128 ? 1 : 2) mlstm_chunk_kernel(MlstmParams<bf16> p, MlstmGates g) {
  constexpr int CH = DK / 8, COLS = kMWarps * 16, VCH = COLS / 8, NT = 32 * (kMWarps + 1);
  constexpr int TILE = kMC * DK * 2, STAGE = 2 * TILE + kMC * COLS * 2 + 3 * kMC * 4 + 64;
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool keeper = warp == kMWarps;
  const int c0 = blockIdx.x * COLS, dk = p.dk;
  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q[b], n_all = p.cu_q[b + 1] - row0, slot = p.slots[b];
  if (n_all <= 0 || slot < 0) return;
  const bool fresh = p.kv_lens[b] == n_all;
  const bool works = keeper ? blockIdx.x == 0 : c0 + warp * 16 < p.dv;
  const int64_t sh = (int64_t)slot * p.H + h;
  float* S = p.state + sh * dk * p.dvp;
  float* N = p.norm + sh * dk;
  const int vrow = c0 + warp * 16 + (lane >> 2), kc = (lane & 3) * 2;
  float acc[DK / 8][4];              // S^T: rows (value columns) lane / 4, + 8; key channels 8 nt + kc, + 1
#pragma unroll
  for (int nt = 0; nt < DK / 8; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = nt * 8 + kc + (e & 1), v = vrow + (e >> 1) * 8;
      float x = 0.f;
      if (works && !fresh && c < dk) {
        if (keeper) x = (lane < 4 && e < 2) ? N[c] : 0.f;
        else if (v < p.dv) x = S[(int64_t)c * p.dvp + v];
      }
      acc[nt][e] = x;
    }
  const int chunks = (n_all + kMC - 1) / kMC;
  const float* before = g.before + (int64_t)h * g.chunks + row0 / kMC + b;
  const int64_t gate_at = (int64_t)h * g.rows + row0;
  const auto load = [&](int j) {
    if (j < chunks) {
      const uint32_t st = sb + (j % kMStages) * STAGE;
      const int t0 = j * kMC;
      const int64_t row = (int64_t)(row0 + t0) * p.ld;
      for (int i = tid; i < kMC * CH; i += NT) {
        const int r = i / CH, c = i % CH;
        const bool ok = t0 + r < n_all && c * 8 < dk;
        const int64_t go = ok ? row + r * p.ld + (int64_t)h * dk + c * 8 : 0;
        cp_async16(st + swz<CH>(r, c), p.q + go, ok);
        cp_async16(st + TILE + swz<CH>(r, c), p.k + go, ok);
      }
      for (int i = tid; i < kMC * VCH; i += NT) {
        const int r = i / VCH, c = i % VCH;
        const bool ok = t0 + r < n_all && c0 + c * 8 < p.dv;
        cp_async16(st + 2 * TILE + swz<VCH>(r, c), p.v + (ok ? row + r * p.ld + (int64_t)h * p.dv + c0 + c * 8 : 0), ok);
      }
      float* gs = reinterpret_cast<float*>(smem + (j % kMStages) * STAGE + 2 * TILE + kMC * COLS * 2);
      if (tid < 3 * kMC) {
        const int which = tid / kMC, t = tid % kMC;
        const float* src = which == 0 ? g.a : (which == 1 ? g.b : g.em);
        gs[tid] = t0 + t < n_all ? src[gate_at + t0 + t] : 0.f;
      } else if (tid == 3 * kMC) {
        gs[tid] = before[j];
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < kMStages - 1; ++s) load(s);
  const int arow = (lane & 7) + (((lane >> 3) & 1) << 3), acb = lane >> 4;
  const int brow = (lane & 7) + ((lane >> 4) << 3), bcb = (lane >> 3) & 1;
  const float qs = p.q_scale;
  for (int j = 0; j < chunks; ++j) {
    const int n = min(kMC, n_all - j * kMC);
    cp_async_wait<kMStages - 2>();
    __syncthreads();                 // chunk j is here, and everybody is done with chunk j - 1, whose stage is filled next
    load(j + kMStages - 1);
    if (!works) continue;
    const uint32_t sq = sb + (j % kMStages) * STAGE, sk = sq + TILE, sv = sk + TILE;
    const float* gs = reinterpret_cast<const float*>(smem + (j % kMStages) * STAGE + 2 * TILE + kMC * COLS * 2);
    const float m_before = gs[3 * kMC], b_last = gs[kMC + n - 1];
    float o[2][4], ol[2][4], pw[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][e] = ol[i][e] = pw[i][e] = 0.f;
    // ---- O^T = S^T Q^T and P = Q K^T
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t qb[4], kb[4], hi[4], lo[4];
      ldmatrix_x4(qb[0], qb[1], qb[2], qb[3], sq + swz<CH>(brow, kk * 2 + bcb));
      ldmatrix_x4(kb[0], kb[1], kb[2], kb[3], sk + swz<CH>(brow, kk * 2 + bcb));
      split_pack(acc[2 * kk][0], acc[2 * kk][1], hi[0], lo[0]);
      split_pack(acc[2 * kk][2], acc[2 * kk][3], hi[1], lo[1]);
      split_pack(acc[2 * kk + 1][0], acc[2 * kk + 1][1], hi[2], lo[2]);
      split_pack(acc[2 * kk + 1][2], acc[2 * kk + 1][3], hi[3], lo[3]);
      const uint32_t qa[4] = {qb[0], qb[2], qb[1], qb[3]};
      mma_bf16_16816(o[0], hi, qb[0], qb[1]);
      mma_bf16_16816(o[1], hi, qb[2], qb[3]);
      mma_bf16_16816(pw[0], qa, kb[0], kb[1]);
      mma_bf16_16816(pw[1], qa, kb[2], kb[3]);
      mma_bf16_16816(ol[0], lo, qb[0], qb[1]);
      mma_bf16_16816(ol[1], lo, qb[2], qb[3]);
    }
    // ---- weights: tokens 8 i + kc (+ 1) of this lane as columns, lane / 4 (+ 8) as rows
    float av[2][2];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = 8 * i + kc + e;
        av[i][e] = gs[t];
        const float f = qs * expf(gs[kMC + t] + m_before);
        o[i][e] = (o[i][e] + ol[i][e]) * f;
        o[i][e + 2] = (o[i][e + 2] + ol[i][e + 2]) * f;
      }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = (lane >> 2) + 8 * u;
      const float bt = gs[kMC + t];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          pw[i][2 * u + e] = 8 * i + kc + e <= t ? pw[i][2 * u + e] * (qs * expf(bt + av[i][e])) : 0.f;
    }
    // ---- O^T += V^T P^T
    uint32_t va[4];
    if (keeper) {
      va[0] = va[2] = lane < 4 ? 0x3F803F80u : 0u;
      va[1] = va[3] = 0u;
    } else {
      ldmatrix_x4_trans(va[0], va[2], va[1], va[3], sv + swz<VCH>(arow, warp * 2 + acb));
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      uint32_t h0, h1, l0, l1;
      split_pack(pw[0][2 * u], pw[0][2 * u + 1], h0, l0);
      split_pack(pw[1][2 * u], pw[1][2 * u + 1], h1, l1);
      mma_bf16_16816(o[u], va, h0, h1);
      mma_bf16_16816(o[u], va, l0, l1);
    }
    // ---- S^T <- keep S^T + (w V)^T K
    uint32_t wh[4], wl[4];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 8 * i + kc;
      const float w0 = t < n ? expf(b_last + av[i][0]) : 0.f, w1 = t + 1 < n ? expf(b_last + av[i][1]) : 0.f;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float2 x = unpack2(va[2 * i + u]);
        split_pack(x.x * w0, x.y * w1, wh[2 * i + u], wl[2 * i + u]);
      }
    }
    const float keep = expf(b_last + m_before);
#pragma unroll
    for (int nt = 0; nt < DK / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[nt][e] *= keep;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t kt[4];
      ldmatrix_x4_trans(kt[0], kt[1], kt[2], kt[3], sk + swz<CH>(arow, kk * 2 + acb));
      mma_bf16_16816(acc[2 * kk], wh, kt[0], kt[1]);
      mma_bf16_16816(acc[2 * kk + 1], wh, kt[2], kt[3]);
      mma_bf16_16816(acc[2 * kk], wl, kt[0], kt[1]);
      mma_bf16_16816(acc[2 * kk + 1], wl, kt[2], kt[3]);
    }
    const int64_t row = row0 + j * kMC;
    if (keeper) {
      if (lane < 4) {
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = 8 * i + kc + e;
            if (t < n) p.div[(row + t) * p.H + h] = fmaxf(fabsf(o[i][e]), gs[2 * kMC + t]) + kDivEps;
          }
      }
      continue;
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = 8 * i + kc + (e & 1), v = vrow + (e >> 1) * 8;
        if (t < n && v < p.dv) p.o[((row + t) * p.H + h) * p.dv + v] = o[i][e];
      }
  }
  cp_async_wait<0>();
  if (!works) return;
#pragma unroll
  for (int nt = 0; nt < DK / 8; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = nt * 8 + kc + (e & 1), v = vrow + (e >> 1) * 8;
      if (c >= dk) continue;
      if (keeper) {
        if (lane < 4 && e < 2) N[c] = acc[nt][e];
      } else if (v < p.dvp) {
        S[(int64_t)c * p.dvp + v] = acc[nt][e];
      }
    }
}

template <int DK>
static int launch_mlstm_chunk(const MlstmParams<bf16>& p, const MlstmGates& g, int n_seqs, cudaStream_t s) {
  constexpr int COLS = kMWarps * 16;
  const size_t smem = (size_t)kMStages * (2 * kMC * DK * 2 + kMC * COLS * 2 + 3 * kMC * 4 + 64);
  const cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  launch_pdl(mlstm_gates_kernel, dim3(p.H, n_seqs), dim3(256), 0, s, p, g);
  const int rc = XLLM_LAUNCH_CHECK();
  if (rc != 0) return rc;
  launch_pdl(mlstm_chunk_kernel<DK>, dim3((p.dv + COLS - 1) / COLS, p.H, n_seqs), dim3(32 * (kMWarps + 1)), smem, s, p, g);
  return XLLM_LAUNCH_CHECK();
}

template <typename T, int V, int J>
static int launch_mlstm_prefill(const MlstmParams<T>& p, int n_seqs, cudaStream_t s) {
  constexpr int COLS = kMlstmWarps * kRecCols;
  const size_t smem = (size_t)kRecTile * (2 * 32 * J + COLS) * 4;
  const cudaError_t e = cudaFuncSetAttribute(mlstm_prefill_kernel<T, V, J>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  launch_pdl(mlstm_prefill_kernel<T, V, J>, dim3((p.dv + COLS - 1) / COLS, p.H, n_seqs), dim3(32 * (kMlstmWarps + 1)), smem, s, p);
  const int rc = XLLM_LAUNCH_CHECK();
  if (rc != 0) return rc;
  launch_pdl(mlstm_top_kernel<T>, dim3(p.H, n_seqs), dim3(256), 0, s, p);
  return XLLM_LAUNCH_CHECK();
}

template <typename T, int V>
static int run_mlstm_prefill(const MlstmParams<T>& p, int n_seqs, cudaStream_t s) {
  if (p.dk <= 32) return launch_mlstm_prefill<T, V, 1>(p, n_seqs, s);
  if (p.dk <= 64) return launch_mlstm_prefill<T, V, 2>(p, n_seqs, s);
  if (p.dk <= 128) return launch_mlstm_prefill<T, V, 4>(p, n_seqs, s);
  if (p.dk <= 256) return launch_mlstm_prefill<T, V, 8>(p, n_seqs, s);
  return launch_mlstm_prefill<T, V, 16>(p, n_seqs, s);
}

}  // namespace xllm

// dtype: 0 bf16, 1 fp32 (projection rows, weights, finished rows).
//   state fp32 [slots, H, dk, dvp], dvp = dv rounded up to 4;  norm fp32 [slots, H, dk];  top fp32 [slots, H]
//   q, k, v: column blocks of rows with stride ld;  zi, zf fp32 with row stride z_ld
// mode 0: one token per sequence (sequence s is row s): gate, norm_w, out are used; dk <= 256, dv <= 128
// mode 1: prompt rows by cu_q: sums to o fp32 [rows, H, dv], denominators to div fp32 [rows, H];  dk <= 512
// mode 2: the same in chunks of 16 tokens (bf16, dk and dv multiples of 8, dk <= 256, aligned rows; otherwise mode 1);
//         gates: fp32 scratch of 3 H rows + H (rows / 16 + n_seqs + 1)
XLLM_API int xllm_mlstm(void* state, void* norm, void* top, const void* slots, const void* cu_q, const void* kv_lens,
                        const void* q, const void* k, const void* v, int64_t ld, const void* zi, const void* zf, int64_t z_ld,
                        const void* gate, int64_t gate_ld, const void* norm_w, void* out, int64_t out_ld, void* o, void* div,
                        void* gates, int rows, int n_seqs, int H, int dk, int dv, float q_scale, float cap, float eps, int dtype, int mode,
                        void* stream) {
  using namespace xllm;
  if (n_seqs == 0) return 0;
  if (H <= 0 || dk <= 0 || dk > 512 || dv <= 0 || !(cap > 0.f)) return (int)cudaErrorInvalidValue;
  if (mode == 0 && (dk > 256 || dv > 128)) return (int)cudaErrorInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  int rc = 0;
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    MlstmParams<T> p;
    p.state = (float*)state; p.norm = (float*)norm; p.top = (float*)top; p.slots = (const int32_t*)slots;
    p.cu_q = (const int32_t*)cu_q; p.kv_lens = (const int32_t*)kv_lens; p.q = (const T*)q; p.k = (const T*)k; p.v = (const T*)v;
    p.ld = ld; p.zi = (const float*)zi; p.zf = (const float*)zf; p.z_ld = z_ld; p.gate = (const T*)gate; p.gate_ld = gate_ld;
    p.norm_w = (const T*)norm_w; p.out = (T*)out; p.out_ld = out_ld; p.o = (float*)o; p.div = (float*)div; p.H = H; p.dk = dk;
    p.dv = dv; p.dvp = (dv + 3) & ~3; p.q_scale = q_scale; p.cap = cap; p.eps = eps;
    if (mode == 0) {
      const int RG = 256 / (p.dvp >> 2), nr = (dk + RG - 1) / RG;
      const size_t smem = (size_t)(2 * ((dk + 3) & ~3) + p.dvp + RG * p.dvp) * 4;
      const dim3 grid(H, n_seqs), block(256);
      if (nr <= 4) launch_pdl(mlstm_decode_kernel<T, 4>, grid, block, smem, s, p);
      else if (nr <= 8) launch_pdl(mlstm_decode_kernel<T, 8>, grid, block, smem, s, p);
      else if (nr <= 16) launch_pdl(mlstm_decode_kernel<T, 16>, grid, block, smem, s, p);
      else launch_pdl(mlstm_decode_kernel<T, 32>, grid, block, smem, s, p);
      rc = XLLM_LAUNCH_CHECK();
      return;
    }
    if constexpr (sizeof(T) == 2) {
      const auto a16 = [](const void* x) { return (((uintptr_t)x) & 15) == 0; };
      if (mode == 2 && gates != nullptr && dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && ld % 8 == 0 && a16(q) && a16(k) && a16(v)) {
        MlstmGates g;
        g.rows = rows; g.chunks = rows / kMC + n_seqs + 1;
        g.a = (float*)gates; g.b = g.a + (int64_t)H * rows; g.em = g.b + (int64_t)H * rows; g.before = g.em + (int64_t)H * rows;
        if (dk <= 64) rc = launch_mlstm_chunk<64>(p, g, n_seqs, s);
        else if (dk <= 128) rc = launch_mlstm_chunk<128>(p, g, n_seqs, s);
        else rc = launch_mlstm_chunk<256>(p, g, n_seqs, s);
        return;
      }
    }
    const auto al = [](const void* x) { return (((uintptr_t)x) & (4 * sizeof(T) - 1)) == 0; };
    if (dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && al(q) && al(k) && al(v)) rc = run_mlstm_prefill<T, 4>(p, n_seqs, s);
    else rc = run_mlstm_prefill<T, 1>(p, n_seqs, s);
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return rc;
}
