// Linear attention with a decaying matrix state, per head:
//
//   S_t = diag(a_t) S_{t-1} + k_t v_t^T        o_t = S_t^T q_t        S [dk, dv] fp32, one per state slot
//
// The decay a_t is either one constant per head (retention) or a value per token and key channel,
// a = sigmoid(W_2 r + b)^(1 / tau) with r the low-rank column block of the projection row (gated linear attention).
// q and k may be rotated (rotate-half or interleaved pairs) and scaled; the output of a head may be divided by its
// root mean square, weighted, and multiplied by silu(g); q, k and v may pass through silu first.  All of that happens
// here, in fp32, from the projection rows as the GEMM left them.
//
//   linattn_decode_kernel     one token per sequence: state read once and written once, output finished (norm, gate)
//   linattn_chunk_kernel      prompt chunks, bf16, dk <= 256: 16 tokens at a time on the tensor cores.  A warp owns 16
//                             state columns for all of dk as fp32 accumulators of S^T, which are the B operand of
//                             O = Q S and the accumulator of S^T += V^T K without leaving the registers.  Every fp32
//                             operand (q and k with their decays, S, the token-token weights) enters the bf16
//                             products as a sum of two bf16 terms, so the recurrence keeps about 16 bits of
//                             significand per operand and accumulates in fp32.
//   linattn_recurrent_kernel  prompt chunks of any dtype and size, token by token in fp32
// (head_norm.cu finishes the fp32 outputs of the two prompt kernels)
//
// A sequence whose rows in the batch are its first tokens (kv_len == number of rows) starts from S = 0 whatever its
// slot holds; slot < 0 marks padding rows.  Token by token a state is decayed as S + (a - 1) S with a - 1 = expm1(log a): a
// itself, rounded to fp32, would be off by 2^-25, which a slow decay multiplies by the 1 / (1 - a) tokens it sums over.  The reference has no such layer; its nearest relative is the Triton
// gated delta rule (xllm/python/kernels_cuda/triton/gdn_prefill.py).  Built without fast-math: errors of the decay
// accumulate over a sequence.
#include "attn_common.cuh"
#include "vec_io.cuh"

namespace xllm {

template <typename T>
struct LinAttnParams {
  float* state;              // [slots, H, dk, dv_pad]
  const int32_t* slots;      // [n_seqs]
  const int32_t* cu_q;       // [n_seqs + 1] token rows (null: sequence s is row s)
  const int32_t* kv_lens;    // [n_seqs]
  const T *q, *k, *v, *g, *r;
  int64_t ld;                // row stride of q, k, v, g, r
  const float* cos_sin;      // [max_pos, rot]: cos | sin; null: no rotation
  const int64_t* positions;  // [T]
  int64_t max_pos;
  const float* log_decay;    // [H], or null: channel decay
  const T* a2;               // [H * dk, rank]
  const T* a2_b;             // [H * dk]
  const T* norm_w;           // [dv] or null
  void* out;                 // decode: T [rows, out_ld], or with raw_out float [rows, H, dv]; prompt: float [T, H, dv]
  int64_t out_ld;
  int n_seqs, H, dk, dv, dv_pad, rot, interleaved, rank, unit_norm, vec_ok;
  int in_silu, raw_out;      // q, k and v pass through silu; decode leaves raw fp32 outputs
  float q_scale, k_scale, inv_tau, eps;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu_f32(float z) { return z / (1.f + expf(-z)); }
// for rows that leave as bf16: hardware exponential and division (2^-21 relative)
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// a projected value as it enters the recurrence
template <typename T>
__device__ __forceinline__ float entering(T x, int in_silu) {
  const float u = to_f32(x);
  return in_silu ? silu_as<T>(u) : u;
}

// element i of a head after the rotation of its first `rot` elements; `cs` is the position's cos | sin row
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int i, int rot, int interleaved, const float* cs, int in_silu) {
  const float u = entering(x[i], in_silu);
  if (cs == nullptr || i >= rot) return u;
  const int half = rot >> 1;
  const bool first = interleaved ? (i & 1) == 0 : i < half;
  const int n = interleaved ? i >> 1 : (first ? i : i - half);
  const int j = interleaved ? i ^ 1 : (first ? i + half : i - half);
  const float v = entering(x[j], in_silu);
  const float c = cs[n], s = cs[half + n];
  return first ? u * c - v * s : u * c + v * s;
}

// log of the decay of channel i of head h for one token (channel decay)
template <typename T>
__device__ __forceinline__ float channel_log_decay(const LinAttnParams<T>& p, const T* r, int64_t c) {
  float z = to_f32(p.a2_b[c]);
  const T* w = p.a2 + c * p.rank;
  for (int j = 0; j < p.rank; ++j) z += to_f32(r[j]) * to_f32(w[j]);
  return log_sigmoid(z) * p.inv_tau;
}

template <typename T>
__device__ __forceinline__ const float* rope_row(const LinAttnParams<T>& p, int64_t t) {
  if (p.cos_sin == nullptr) return nullptr;
  int64_t pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
  return p.cos_sin + pos * p.rot;
}

// ------------------------------------------------------------------------------------------------ decode
// grid (heads, sequences), 256 threads: dv_pad / 4 column groups x row groups; a thread updates every RG-th row of its
// four columns, NR rows in flight at a time.
template <typename T, int NR>
__global__ void __launch_bounds__(256) linattn_decode_kernel(LinAttnParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  const int dk = p.dk, dv = p.dv, dvp = p.dv_pad;
  const int dkp = (dk + 3) & ~3;          // 16-byte aligned sections
  float* qs = sm;
  float* ks = qs + dkp;
  float* as = ks + dkp;
  float* vs = as + dkp;                   // [dvp]
  float* red = vs + dvp;                  // [RG][dvp]
  __shared__ float red32[32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int CG = dvp >> 2, RG = 256 / CG;
  const int cg = tid % CG, rg = tid / CG;
  pdl_wait();
  pdl_launch_dependents();
  T* orow = reinterpret_cast<T*>(p.out) + b * p.out_ld + (int64_t)h * dv;
  float* raw = reinterpret_cast<float*>(p.out) + ((int64_t)b * p.H + h) * dv;
  const int slot = p.slots[b];
  const int len = p.kv_lens[b];
  if (slot < 0 || len <= 0) {
    for (int i = tid; i < dv; i += 256) {
      if (p.raw_out) raw[i] = 0.f;
      else orow[i] = from_f32<T>(0.f);
    }
    return;
  }
  const bool active = rg < RG, fresh = len == 1;
  float* S = p.state + (((int64_t)slot * p.H + h) * dk) * dvp + cg * 4;
  float4 s[NR];
  const auto fetch = [&](int base) {
#pragma unroll
    for (int u = 0; u < NR; ++u) {
      const int r = base + u * RG;
      s[u] = (active && !fresh && r < dk) ? *reinterpret_cast<const float4*>(S + (int64_t)r * dvp)
                                          : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  fetch(rg);
  {
    const T* qr = p.q + b * p.ld + (int64_t)h * dk;
    const T* kr = p.k + b * p.ld + (int64_t)h * dk;
    const T* vr = p.v + b * p.ld + (int64_t)h * dv;
    const float* cs = rope_row(p, b);
    for (int i = tid; i < dk; i += 256) {
      qs[i] = rotated(qr, i, p.rot, p.interleaved, cs, p.in_silu) * p.q_scale;
      ks[i] = rotated(kr, i, p.rot, p.interleaved, cs, p.in_silu) * p.k_scale;
      as[i] = expm1f(p.log_decay != nullptr ? p.log_decay[h]
                                          : channel_log_decay(p, p.r + b * p.ld, (int64_t)h * dk + i));
    }
    for (int i = tid; i < dvp; i += 256) vs[i] = i < dv ? entering(vr[i], p.in_silu) : 0.f;
  }
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    const float4 v4 = *reinterpret_cast<const float4*>(vs + cg * 4);
    for (int base = rg; base < dk; base += NR * RG) {
      if (base != rg) fetch(base);
#pragma unroll
      for (int u = 0; u < NR; ++u) {
        const int r = base + u * RG;
        if (r >= dk) break;
        const float a = as[r], kk = ks[r], qq = qs[r];
        float4 x = s[u];
        x.x = fmaf(a, x.x, x.x) + kk * v4.x; x.y = fmaf(a, x.y, x.y) + kk * v4.y;
        x.z = fmaf(a, x.z, x.z) + kk * v4.z; x.w = fmaf(a, x.w, x.w) + kk * v4.w;
        *reinterpret_cast<float4*>(S + (int64_t)r * dvp) = x;
        o.x += qq * x.x; o.y += qq * x.y; o.z += qq * x.z; o.w += qq * x.w;
      }
    }
    *reinterpret_cast<float4*>(red + rg * dvp + cg * 4) = o;
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = tid; i < dvp; i += 256) {
    float a = 0.f;
    for (int w = 0; w < RG; ++w) a += red[w * dvp + i];
    if (p.raw_out && i < dv) raw[i] = a;
    vs[i] = a;                            // v is no longer needed; each thread reads back its own entries
    if (i < dv) ss += a * a;
  }
  if (p.raw_out) return;
  float inv = 1.f;
  if (p.unit_norm) inv = 1.f / sqrtf(block_sum(ss, red32) / (float)dv + p.eps);
  for (int i = tid; i < dv; i += 256) {
    float a = vs[i] * inv;
    if (p.norm_w != nullptr) a *= to_f32(p.norm_w[i]);
    if (p.g != nullptr) a *= silu_f32(to_f32(p.g[b * p.ld + (int64_t)h * dv + i]));
    orow[i] = from_f32<T>(a);
  }
}

// ------------------------------------------------------------------------------------------------ token by token
// grid (heads, sequences, column slices of 32), 256 threads: 8 column groups of four x 32 row groups, NR rows each.
template <typename T, int NR>
__global__ void __launch_bounds__(256) linattn_recurrent_kernel(LinAttnParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(16) float vs[2][32];
  __shared__ __align__(16) float red[2][8][32];
  const int dk = p.dk, dvp = p.dv_pad;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int cg = tid & 7, rg = tid >> 3, c0 = blockIdx.z * 32;
  const int col = c0 + cg * 4;
  pdl_wait();
  pdl_launch_dependents();
  const int r0 = p.cu_q[b], n = p.cu_q[b + 1] - r0;
  const int slot = p.slots[b];
  if (n <= 0 || slot < 0) return;
  const bool fresh = p.kv_lens[b] == n, live = col < dvp;
  float* S = p.state + (((int64_t)slot * p.H + h) * dk) * dvp + col;
  float4 s[NR];
#pragma unroll
  for (int u = 0; u < NR; ++u) {
    const int r = rg + 32 * u;
    s[u] = (live && !fresh && r < dk) ? *reinterpret_cast<const float4*>(S + (int64_t)r * dvp)
                                      : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float* out = reinterpret_cast<float*>(p.out);
  for (int t = 0; t < n; ++t) {
    const int64_t row = r0 + t;
    float* qs = sm + (t & 1) * 3 * dk;
    float* ks = qs + dk;
    float* as = ks + dk;
    const T* qr = p.q + row * p.ld + (int64_t)h * dk;
    const T* kr = p.k + row * p.ld + (int64_t)h * dk;
    const float* cs = rope_row(p, row);
    for (int i = tid; i < dk; i += 256) {
      qs[i] = rotated(qr, i, p.rot, p.interleaved, cs, p.in_silu) * p.q_scale;
      ks[i] = rotated(kr, i, p.rot, p.interleaved, cs, p.in_silu) * p.k_scale;
      as[i] = expm1f(p.log_decay != nullptr ? p.log_decay[h]
                                          : channel_log_decay(p, p.r + row * p.ld, (int64_t)h * dk + i));
    }
    if (tid < 32) vs[t & 1][tid] = c0 + tid < p.dv ? entering(p.v[row * p.ld + (int64_t)h * p.dv + c0 + tid], p.in_silu) : 0.f;
    __syncthreads();
    const float4 v4 = *reinterpret_cast<const float4*>(&vs[t & 1][cg * 4]);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int u = 0; u < NR; ++u) {
      const int r = rg + 32 * u;
      if (r >= dk) break;
      const float a = as[r], kk = ks[r], qq = qs[r];
      float4& x = s[u];
      x.x = fmaf(a, x.x, x.x) + kk * v4.x; x.y = fmaf(a, x.y, x.y) + kk * v4.y;
      x.z = fmaf(a, x.z, x.z) + kk * v4.z; x.w = fmaf(a, x.w, x.w) + kk * v4.w;
      o.x += qq * x.x; o.y += qq * x.y; o.z += qq * x.z; o.w += qq * x.w;
    }
#pragma unroll
    for (int m = 8; m <= 16; m <<= 1) {
      o.x += __shfl_xor_sync(0xffffffffu, o.x, m);
      o.y += __shfl_xor_sync(0xffffffffu, o.y, m);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, m);
      o.w += __shfl_xor_sync(0xffffffffu, o.w, m);
    }
    if ((tid & 31) < 8) *reinterpret_cast<float4*>(&red[t & 1][tid >> 5][cg * 4]) = o;
    __syncthreads();
    if (tid < 32 && c0 + tid < p.dv) {
      float a = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) a += red[t & 1][w][tid];
      out[(row * p.H + h) * p.dv + c0 + tid] = a;
    }
  }
  if (live) {
#pragma unroll
    for (int u = 0; u < NR; ++u) {
      const int r = rg + 32 * u;
      if (r < dk) *reinterpret_cast<float4*>(S + (int64_t)r * dvp) = s[u];
    }
  }
}

// ------------------------------------------------------------------------------------------------ chunks of 16 tokens
// A prompt of several segments runs as three launches: the state every segment adds on its own (STATE_ONLY, from zero),
// a scan over the segments' states, and the outputs of all segments side by side, each from its start state.  A prompt
// of one segment needs the last launch only.
constexpr int kLC = 16;                     // tokens per chunk
constexpr float kLogRange = 86.f;           // |log2 decay| between a chunk's ends and its reference token

struct SegParams {
  float* state;      // [slot][H][dk][dv_pad]: local states, then (after the scan) start states; null: one segment
  float* decay;      // [slot][H][dk]: decay over a segment
  int len;           // tokens per segment (multiple of 16)
  void* fused_out;   // bf16 [T, out_ld], finished rows (dv fits one CTA), or null: raw fp32 to out
  int64_t out_ld;
};

// slots of the segments of sequence b: unique because a sequence of n rows has at most n / len + 1 whole segments
__device__ __forceinline__ int64_t seg_slot(int row0, int b, int s, int len) { return (int64_t)row0 / len + b + s; }

template <int DK, int NW>
struct ChunkSmem {
  static constexpr int VC = NW * 16;        // value columns per CTA
  static constexpr int VCP = VC < 64 ? 64 : VC;
  static constexpr int tile = kLC * DK * 2, vtile = kLC * VCP * 2;
  static constexpr int khi = 0, klo = tile, qhi = 2 * tile, qlo = 3 * tile;
  static constexpr int v = 4 * tile;                       // 2 x [16][VCP] swizzled
  static constexpr int g = v + 2 * vtile;                  // 2 x [16][VCP] plain
  static constexpr int raw = g + 2 * vtile;                // 2 x (q, k) [16][DK]
  static constexpr int fs = raw + 4 * tile;                // [DK] scale of the state rows
  static constexpr int et = fs + DK * 4;                   // [DK] decay from the reference token to the chunk's end
  static constexpr int tot = et + DK * 4;                  // [DK] log2 decay over the segment so far
  static constexpr int ssm = tot + DK * 4;                 // [16][NW] partial sums of squares
  static constexpr int dyn = ssm + NW * kLC * 4;
  // dyn: cos | sin 2 x [16][rot] fp32; channel decay: lw [16][DK] fp32, bias [DK], raw r 2 x [16][RP], a2 [DK][RP + 8]
};

template <int DK, int NW, bool STATE_ONLY>
__global__ void __launch_bounds__(NW * 32, DK > 128 ? 1 : 512 / (NW * 32)) linattn_chunk_kernel(LinAttnParams<bf16> p, SegParams sp) {
  using L = ChunkSmem<DK, NW>;
  constexpr int CH = DK / 8, VCH = L::VCP / 8, NT = NW * 32;
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.x, b = blockIdx.y;
  const int slices = (p.dv + L::VC - 1) / L::VC;
  const int seg = blockIdx.z / slices, c0 = (blockIdx.z - seg * slices) * L::VC;
  const int dk = p.dk, rot = p.cos_sin != nullptr ? p.rot : 0;
  const bool channel = p.log_decay == nullptr;
  const int RP = channel ? (p.rank + 15) & ~15 : 0, A2S = RP + 8;
  float* fs = reinterpret_cast<float*>(smem + L::fs);
  float* et = reinterpret_cast<float*>(smem + L::et);
  float* tot = reinterpret_cast<float*>(smem + L::tot);
  float* ssm = reinterpret_cast<float*>(smem + L::ssm);
  float* csb = reinterpret_cast<float*>(smem + L::dyn);                       // [2][16][rot]
  float* lw = csb + 2 * kLC * rot;                                            // [16][DK]
  float* bias = lw + (channel ? kLC * DK : 0);
  bf16* rb = reinterpret_cast<bf16*>(bias + (channel ? DK : 0));              // [2][16][RP]
  bf16* a2s = rb + 2 * kLC * RP;                                              // [DK][A2S]
  __shared__ float elog[2 * kLC];
  pdl_wait();
  pdl_launch_dependents();
  const int row_first = p.cu_q[b], n_seq = p.cu_q[b + 1] - row_first;
  const int slot = p.slots[b];
  if (n_seq <= 0 || slot < 0 || seg * sp.len >= n_seq) return;
  const int row0 = row_first + seg * sp.len, n_all = min(sp.len, n_seq - seg * sp.len);
  const bool one_seg = sp.state == nullptr;
  const bool fresh = STATE_ONLY || (one_seg && p.kv_lens[b] == n_seq);
  const float lg = channel ? 0.f : fmaxf(p.log_decay[h], -1e4f) * 1.44269504088896341f;    // log2 of the constant decay

  // ---- state columns of this warp: acc[nt] holds S^T rows (value columns) lane/4, +8 and key channels nt*8 + ..
  float acc[DK / 8][4];
  const int vrow = c0 + warp * 16 + (lane >> 2);
  const bool has_cols = c0 + warp * 16 < p.dv;
  const int64_t seg_at = one_seg ? 0 : seg_slot(row_first, b, seg, sp.len) * p.H + h;
  float* S = one_seg ? p.state + (((int64_t)slot * p.H + h) * dk) * p.dv_pad : sp.state + seg_at * dk * p.dv_pad;
#pragma unroll
  for (int nt = 0; nt < DK / 8; ++nt) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = nt * 8 + (lane & 3) * 2 + (e & 1), v = vrow + (e >> 1) * 8;
      acc[nt][e] = (!fresh && c < dk && v < p.dv) ? S[(int64_t)c * p.dv_pad + v] : 0.f;
    }
  }
  for (int i = tid; i < DK; i += NT) {
    et[i] = 1.f;
    tot[i] = 0.f;
    if (channel) bias[i] = i < dk ? __bfloat162float(p.a2_b[(int64_t)h * dk + i]) : 0.f;
  }
  if (channel) {
    for (int i = tid; i < DK * RP; i += NT) {
      const int c = i / RP, j = i - c * RP;
      a2s[c * A2S + j] = (c < dk && j < p.rank) ? p.a2[((int64_t)h * dk + c) * p.rank + j] : __float2bfloat16(0.f);
    }
  } else {
    if (tid < 2 * kLC) elog[tid] = exp2f((float)(tid - kLC) * lg);      // elog[16 + i] = decay^i
  }

  const int64_t last_pos = p.max_pos - 1;
  const int64_t pos0 = rot > 0 ? max((int64_t)0, min(p.positions[row0], last_pos)) : 0;
  const auto load_raw = [&](int t0, int buf) {              // 16 token rows from t0 (of this segment)
    const uint32_t raws = sb + L::raw + buf * 2 * L::tile, vsm = sb + L::v + buf * L::vtile, gsm = sb + L::g + buf * L::vtile;
    const int64_t base = (int64_t)(row0 + t0);
    const bool gate = !STATE_ONLY && sp.fused_out != nullptr && p.g != nullptr;
    if (p.vec_ok) {
      const int64_t row = base * p.ld;
#pragma unroll
      for (int i = tid; i < kLC * CH; i += NT) {
        const int r = i / CH, c = i % CH;                    // powers of two
        if (c * 8 >= dk) continue;
        const bool ok = t0 + r < n_all;
        const int64_t go = row + (ok ? r : 0) * p.ld + h * dk + c * 8;
        if (!STATE_ONLY) cp_async16(raws + (r * DK + c * 8) * 2, p.q + go, ok);
        cp_async16(raws + L::tile + (r * DK + c * 8) * 2, p.k + go, ok);
      }
#pragma unroll
      for (int i = tid; i < kLC * (L::VC / 8); i += NT) {
        const int r = i / (L::VC / 8), c = i % (L::VC / 8);
        const bool ok = t0 + r < n_all && c0 + c * 8 < p.dv;
        const int64_t go = ok ? row + r * p.ld + h * p.dv + c0 + c * 8 : 0;
        cp_async16(vsm + swz<VCH>(r, c), p.v + go, ok);
        if (gate) cp_async16(gsm + (r * L::VCP + c * 8) * 2, p.g + go, ok);
      }
      if (channel) {
        const int pr = RP >> 3;
        for (int i = tid; i < kLC * pr; i += NT) {
          const int r = i / pr, c = i - r * pr;
          const bool ok = t0 + r < n_all && c * 8 < p.rank;
          cp_async16(smem_u32(rb + (buf * kLC + r) * RP + c * 8), ok ? p.r + row + r * p.ld + c * 8 : p.r, ok);
        }
      }
    } else {
      bf16* rq = reinterpret_cast<bf16*>(smem + L::raw + buf * 2 * L::tile);
      const bf16 zero = __float2bfloat16(0.f);
      for (int i = tid; i < kLC * dk; i += NT) {
        const int r = i / dk, c = i - r * dk;
        const bool ok = t0 + r < n_all;
        const int64_t go = (base + (ok ? r : 0)) * p.ld + (int64_t)h * dk + c;
        rq[r * DK + c] = ok ? p.q[go] : zero;
        rq[kLC * DK + r * DK + c] = ok ? p.k[go] : zero;
      }
      for (int i = tid; i < kLC * L::VC; i += NT) {
        const int r = i / L::VC, c = i - r * L::VC;
        const bool ok = t0 + r < n_all && c0 + c < p.dv;
        const int64_t go = ok ? (base + r) * p.ld + (int64_t)h * p.dv + c0 + c : 0;
        *reinterpret_cast<bf16*>(smem + L::v + buf * L::vtile + swz<VCH>(r, c >> 3) + (c & 7) * 2) = ok ? p.v[go] : zero;
        if (gate) reinterpret_cast<bf16*>(smem + L::g + buf * L::vtile)[r * L::VCP + c] = ok ? p.g[go] : zero;
      }
      for (int i = tid; i < kLC * RP; i += NT) {
        const int r = i / RP, c = i - r * RP;
        const bool ok = t0 + r < n_all && c < p.rank;
        rb[(buf * kLC + r) * RP + c] = ok ? p.r[(base + r) * p.ld + c] : zero;
      }
    }
    if (rot > 0) {
      if (rot % 4 == 0) {
#pragma unroll
        for (int i = tid; i < kLC * (DK / 4); i += NT) {
          const int r = i / (DK / 4), c = i % (DK / 4);
          if (c * 4 >= rot) continue;
          const int64_t pos = min(pos0 + t0 + r, last_pos);   // the rows of a sequence are consecutive positions
          cp_async16(smem_u32(csb + (buf * kLC + r) * rot + c * 4), p.cos_sin + pos * rot + c * 4, t0 + r < n_all);
        }
      } else {
        for (int i = tid; i < kLC * rot; i += NT) {
          const int r = i / rot, c = i - r * rot;
          csb[(buf * kLC + r) * rot + c] = t0 + r < n_all ? rope_row(p, base + r)[c] : 0.f;
        }
      }
    }
    cp_async_commit();
  };
  const float inv_dv = 1.f / (float)p.dv;
  const bool by_four = dk % 4 == 0 && rot % 4 == 0;       // four channels of a token at a time

  load_raw(0, 0);
  int buf = 0;
  for (int t0 = 0; t0 < n_all; t0 += kLC, buf ^= 1) {
    const int n = min(kLC, n_all - t0);
    cp_async_wait<0>();
    __syncthreads();                       // the raw tiles are here, and nobody reads the operand tiles any more
    if (t0 + kLC < n_all) load_raw(t0 + kLC, buf ^ 1);
    const bf16* rq = reinterpret_cast<const bf16*>(smem + L::raw + buf * 2 * L::tile);
    const bf16* rk = rq + kLC * DK;

    // ---- cumulative log2 decays of the chunk (channel decay): z on the tensor cores, the sum over tokens by shuffles
    bool unsafe = false;
    if (channel) {
      const bf16* r = rb + buf * kLC * RP;
      const int ref = n >> 1;
      for (int nt = warp; nt < DK / 8; nt += NW) {
        float z[4];
        const int c = nt * 8 + (lane & 3) * 2;
        z[0] = z[2] = bias[c];
        z[1] = z[3] = bias[c + 1];
        for (int ks = 0; ks < RP; ks += 16) {
          uint32_t a[4];
          const int k0 = ks + (lane & 3) * 2, ra = lane >> 2;
          a[0] = *reinterpret_cast<const uint32_t*>(r + ra * RP + k0);
          a[1] = *reinterpret_cast<const uint32_t*>(r + (ra + 8) * RP + k0);
          a[2] = *reinterpret_cast<const uint32_t*>(r + ra * RP + k0 + 8);
          a[3] = *reinterpret_cast<const uint32_t*>(r + (ra + 8) * RP + k0 + 8);
          const bf16* w = a2s + (nt * 8 + (lane >> 2)) * A2S + k0;
          mma_bf16_16816(z, a, *reinterpret_cast<const uint32_t*>(w), *reinterpret_cast<const uint32_t*>(w + 8));
        }
        const int ta = lane >> 2;
#pragma unroll
        for (int e = 0; e < 4; ++e)
          z[e] = ta + (e >> 1) * 8 < n ? log_sigmoid(z[e]) * (p.inv_tau * 1.44269504088896341f) : 0.f;
#pragma unroll
        for (int d = 4; d < 32; d <<= 1) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float up = __shfl_up_sync(0xffffffffu, z[e], d);
            if (lane >= d) z[e] += up;
          }
        }
        z[2] += __shfl_sync(0xffffffffu, z[0], 28 + (lane & 3));
        z[3] += __shfl_sync(0xffffffffu, z[1], 28 + (lane & 3));
        *reinterpret_cast<float2*>(lw + ta * DK + c) = make_float2(z[0], z[1]);
        *reinterpret_cast<float2*>(lw + (ta + 8) * DK + c) = make_float2(z[2], z[3]);
        const int rl = (ref & 7) * 4 + (lane & 3);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float m0 = __shfl_sync(0xffffffffu, z[e], rl), m1 = __shfl_sync(0xffffffffu, z[e + 2], rl);
          const float m = ref < 8 ? m0 : m1;
          // (the first token's lane, the last token's lane) see the extremes: the sums fall monotonically
          if (c + e < dk && ((lane < 4 && z[e] - m > kLogRange) || (lane >= 28 && m - z[e + 2] > kLogRange))) unsafe = true;
        }
      }
    } else {
      unsafe = -lg * (float)kLC > kLogRange;
    }
    unsafe = __syncthreads_or(unsafe);
    // decays that span more than fp32 can hold against one reference token: one token at a time
    const int step = unsafe ? 1 : n;
    for (int s0 = 0; s0 < n; s0 += step) {
      const int s1 = s0 + step, ref = s0 + (step >> 1);
      if (s0 > 0) __syncthreads();
      // ---- operand tiles: q and k rotated, scaled, and multiplied by their decay against token `ref`
      if (by_four) {
        const int half = rot >> 1, r4 = rot >> 2;
        for (int i = tid; i < kLC * (DK / 4); i += NT) {
          const int t = i / (DK / 4), m = i - t * (DK / 4);
          const bool turns = m < r4, split = turns && !p.interleaved;
          const int ca = split ? 2 * m : 4 * m, cb = split ? 2 * m + half : 4 * m + 2;     // two channels each
          float k4[4] = {0.f, 0.f, 0.f, 0.f}, q4[4] = {0.f, 0.f, 0.f, 0.f};
          if (t >= s0 && t < s1 && 4 * m < dk) {
            const float2 ka = unpack2(*reinterpret_cast<const uint32_t*>(rk + t * DK + ca));
            const float2 kb = unpack2(*reinterpret_cast<const uint32_t*>(rk + t * DK + cb));
            k4[0] = ka.x; k4[1] = ka.y; k4[2] = kb.x; k4[3] = kb.y;
            if (!STATE_ONLY) {
              const float2 qa = unpack2(*reinterpret_cast<const uint32_t*>(rq + t * DK + ca));
              const float2 qb = unpack2(*reinterpret_cast<const uint32_t*>(rq + t * DK + cb));
              q4[0] = qa.x; q4[1] = qa.y; q4[2] = qb.x; q4[3] = qb.y;
            }
            if (p.in_silu) {
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                k4[e] = silu_fast(k4[e]);
                if (!STATE_ONLY) q4[e] = silu_fast(q4[e]);
              }
            }
            if (turns) {
              const float* cs = csb + (buf * kLC + t) * rot;
              const float2 co = *reinterpret_cast<const float2*>(cs + 2 * m);
              const float2 si = *reinterpret_cast<const float2*>(cs + half + 2 * m);
              const auto turn = [&](float* x) {
                const float x0 = x[0], x1 = x[1], x2 = x[2], x3 = x[3];
                if (split) {                 // partners (0, 2) and (1, 3)
                  x[0] = x0 * co.x - x2 * si.x; x[2] = x2 * co.x + x0 * si.x;
                  x[1] = x1 * co.y - x3 * si.y; x[3] = x3 * co.y + x1 * si.y;
                } else {                     // partners (0, 1) and (2, 3)
                  x[0] = x0 * co.x - x1 * si.x; x[1] = x1 * co.x + x0 * si.x;
                  x[2] = x2 * co.y - x3 * si.y; x[3] = x3 * co.y + x2 * si.y;
                }
              };
              turn(k4);
              if (!STATE_ONLY) turn(q4);
            }
            if (channel) {
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const int c = (e < 2 ? ca : cb) + (e & 1);
                const float d = lw[t * DK + c] - lw[ref * DK + c];
                k4[e] *= p.k_scale * exp2f(-d);
                if (!STATE_ONLY) q4[e] *= p.q_scale * exp2f(d);
              }
            } else {
              const float fk = p.k_scale * (step == 1 ? 1.f : elog[kLC + ref - t]);
              const float fq = p.q_scale * (step == 1 ? 1.f : elog[kLC + t - ref]);
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                k4[e] *= fk;
                q4[e] *= fq;
              }
            }
          }
          const uint32_t oa = swz<CH>(t, ca >> 3) + (ca & 7) * 2, ob = swz<CH>(t, cb >> 3) + (cb & 7) * 2;
          uint32_t hi, lo;
          split_pack(k4[0], k4[1], hi, lo);
          *reinterpret_cast<uint32_t*>(smem + L::khi + oa) = hi;
          *reinterpret_cast<uint32_t*>(smem + L::klo + oa) = lo;
          split_pack(k4[2], k4[3], hi, lo);
          *reinterpret_cast<uint32_t*>(smem + L::khi + ob) = hi;
          *reinterpret_cast<uint32_t*>(smem + L::klo + ob) = lo;
          if (!STATE_ONLY) {
            split_pack(q4[0], q4[1], hi, lo);
            *reinterpret_cast<uint32_t*>(smem + L::qhi + oa) = hi;
            *reinterpret_cast<uint32_t*>(smem + L::qlo + oa) = lo;
            split_pack(q4[2], q4[3], hi, lo);
            *reinterpret_cast<uint32_t*>(smem + L::qhi + ob) = hi;
            *reinterpret_cast<uint32_t*>(smem + L::qlo + ob) = lo;
          }
        }
      } else {
        for (int i = tid; i < kLC * (DK / 2); i += NT) {
          const int t = i / (DK / 2), c = (i - t * (DK / 2)) * 2;
          float qv[2] = {0.f, 0.f}, kv[2] = {0.f, 0.f};
          if (t >= s0 && t < s1 && c < dk) {
            const float* cs = rot > 0 ? csb + (buf * kLC + t) * rot : nullptr;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              if (c + e >= dk) break;
              float eq = 1.f, ek = 1.f;
              if (channel) {
                const float d = lw[t * DK + c + e] - lw[ref * DK + c + e];
                eq = exp2f(d);
                ek = exp2f(-d);
              } else if (step > 1) {
                eq = elog[kLC + t - ref];
                ek = elog[kLC + ref - t];
              }
              qv[e] = rotated(rq + t * DK, c + e, rot, p.interleaved, cs, p.in_silu) * p.q_scale * eq;
              kv[e] = rotated(rk + t * DK, c + e, rot, p.interleaved, cs, p.in_silu) * p.k_scale * ek;
            }
          }
          uint32_t qh, ql, kh, kl;
          split_pack(qv[0], qv[1], qh, ql);
          split_pack(kv[0], kv[1], kh, kl);
          const uint32_t o = swz<CH>(t, c >> 3) + (c & 7) * 2;
          *reinterpret_cast<uint32_t*>(smem + L::khi + o) = kh;
          *reinterpret_cast<uint32_t*>(smem + L::klo + o) = kl;
          *reinterpret_cast<uint32_t*>(smem + L::qhi + o) = qh;
          *reinterpret_cast<uint32_t*>(smem + L::qlo + o) = ql;
        }
      }
      for (int c = tid; c < DK; c += NT) {
        float lref, lend;                     // log2 decay: state -> reference token, reference token -> end
        if (channel) {
          const float m = lw[ref * DK + c];
          lref = m - (s0 > 0 ? lw[(s0 - 1) * DK + c] : 0.f);
          lend = lw[(s1 - 1) * DK + c] - m;
        } else {
          lref = (float)(ref - s0 + 1) * lg;
          lend = (float)(s1 - 1 - ref) * lg;
        }
        fs[c] = et[c] * exp2f(lref);
        et[c] = exp2f(lend);
        tot[c] += lref + lend;
      }
      __syncthreads();

      // ---- O = Q S + mask(Q K^T) V ;  S^T += V^T K
      const int arow = (lane & 7) + (((lane >> 3) & 1) << 3), acb = lane >> 4;
      float o[2][4];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
      if (has_cols) {
        uint32_t v0, v1, v2, v3;
        ldmatrix_x4_trans(v0, v1, v2, v3, sb + L::v + buf * L::vtile + swz<VCH>(arow, warp * 2 + acb));
        if (p.in_silu) {                    // a value belongs to one warp only
          const auto act = [](uint32_t& u) {
            const float2 f = unpack2(u);
            u = pack_bf162(silu_fast(f.x), silu_fast(f.y));
          };
          act(v0); act(v1); act(v2); act(v3);
        }
        if (!STATE_ONLY) {
          float pw[2][4];
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) pw[j][e] = 0.f;
          const int brow = (lane & 7) + ((lane >> 4) << 3), bcb = (lane >> 3) & 1;
#pragma unroll
          for (int kk = 0; kk < DK / 16; ++kk) {
            uint32_t qh[4], ql[4], kh[4], kl[4];
            const uint32_t ao = swz<CH>(arow, kk * 2 + acb), bo = swz<CH>(brow, kk * 2 + bcb);
            ldmatrix_x4(qh[0], qh[1], qh[2], qh[3], sb + L::qhi + ao);
            ldmatrix_x4(ql[0], ql[1], ql[2], ql[3], sb + L::qlo + ao);
            ldmatrix_x4(kh[0], kh[1], kh[2], kh[3], sb + L::khi + bo);
            ldmatrix_x4(kl[0], kl[1], kl[2], kl[3], sb + L::klo + bo);
            const float2 f0 = *reinterpret_cast<const float2*>(fs + kk * 16 + (lane & 3) * 2);
            const float2 f1 = *reinterpret_cast<const float2*>(fs + kk * 16 + 8 + (lane & 3) * 2);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              float* x = acc[2 * kk] + 2 * j;
              float* y = acc[2 * kk + 1] + 2 * j;
              x[0] *= f0.x; x[1] *= f0.y;
              y[0] *= f1.x; y[1] *= f1.y;
              uint32_t bh0, bl0, bh1, bl1;
              split_pack(x[0], x[1], bh0, bl0);
              split_pack(y[0], y[1], bh1, bl1);
              mma_bf16_16816(o[j], qh, bh0, bh1);
              mma_bf16_16816(pw[j], qh, kh[2 * j], kh[2 * j + 1]);
              mma_bf16_16816(o[j], ql, bh0, bh1);
              mma_bf16_16816(pw[j], ql, kh[2 * j], kh[2 * j + 1]);
              mma_bf16_16816(o[j], qh, bl0, bl1);
              mma_bf16_16816(pw[j], qh, kl[2 * j], kl[2 * j + 1]);
            }
          }
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int s = j * 8 + (lane & 3) * 2 + (e & 1), t = (lane >> 2) + (e >> 1) * 8;
              if (s > t) pw[j][e] = 0.f;
            }
          uint32_t pa[4], pb[4];
          split_pack(pw[0][0], pw[0][1], pa[0], pb[0]);
          split_pack(pw[0][2], pw[0][3], pa[1], pb[1]);
          split_pack(pw[1][0], pw[1][1], pa[2], pb[2]);
          split_pack(pw[1][2], pw[1][3], pa[3], pb[3]);
          mma_bf16_16816(o[0], pa, v0, v1);
          mma_bf16_16816(o[1], pa, v2, v3);
          mma_bf16_16816(o[0], pb, v0, v1);
          mma_bf16_16816(o[1], pb, v2, v3);
        } else {
#pragma unroll
          for (int nt = 0; nt < DK / 8; ++nt) {
            const float2 f = *reinterpret_cast<const float2*>(fs + nt * 8 + (lane & 3) * 2);
            acc[nt][0] *= f.x; acc[nt][1] *= f.y; acc[nt][2] *= f.x; acc[nt][3] *= f.y;
          }
        }
        const uint32_t va[4] = {v0, v2, v1, v3};
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          uint32_t kh[4], kl[4];
          const uint32_t ko = swz<CH>(arow, kk * 2 + acb);
          ldmatrix_x4_trans(kh[0], kh[1], kh[2], kh[3], sb + L::khi + ko);
          ldmatrix_x4_trans(kl[0], kl[1], kl[2], kl[3], sb + L::klo + ko);
          mma_bf16_16816(acc[2 * kk], va, kh[0], kh[1]);
          mma_bf16_16816(acc[2 * kk + 1], va, kh[2], kh[3]);
          mma_bf16_16816(acc[2 * kk], va, kl[0], kl[1]);
          mma_bf16_16816(acc[2 * kk + 1], va, kl[2], kl[3]);
        }
      }
      if (STATE_ONLY) continue;
      // ---- rows out: raw, or finished (norm over the head, weight, gate) when this CTA holds all of the head
      if (sp.fused_out == nullptr) {
        if (!has_cols) continue;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; e += 2) {
            const int t = (lane >> 2) + (e >> 1) * 8, c = c0 + warp * 16 + j * 8 + (lane & 3) * 2;
            if (t < s0 || t >= s1 || c >= p.dv) continue;
            float* dst = reinterpret_cast<float*>(p.out) + ((int64_t)(row0 + t0 + t) * p.H + h) * p.dv + c;
            if (p.dv % 2 == 0) {
              *reinterpret_cast<float2*>(dst) = make_float2(o[j][e], o[j][e + 1]);
            } else {
              dst[0] = o[j][e];
              if (c + 1 < p.dv) dst[1] = o[j][e + 1];
            }
          }
        continue;
      }
      if (p.unit_norm) {
        float sa = o[0][0] * o[0][0] + o[0][1] * o[0][1] + o[1][0] * o[1][0] + o[1][1] * o[1][1];
        float sc = o[0][2] * o[0][2] + o[0][3] * o[0][3] + o[1][2] * o[1][2] + o[1][3] * o[1][3];
        sa += __shfl_xor_sync(0xffffffffu, sa, 1);
        sa += __shfl_xor_sync(0xffffffffu, sa, 2);
        sc += __shfl_xor_sync(0xffffffffu, sc, 1);
        sc += __shfl_xor_sync(0xffffffffu, sc, 2);
        if ((lane & 3) == 0) {
          ssm[(lane >> 2) * NW + warp] = sa;
          ssm[((lane >> 2) + 8) * NW + warp] = sc;
        }
        __syncthreads();
      }
      const bf16* gs = reinterpret_cast<const bf16*>(smem + L::g + buf * L::vtile);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int t = (lane >> 2) + u * 8;
        float inv = 1.f;
        if (p.unit_norm) {
          float ss = 0.f;
#pragma unroll
          for (int w = 0; w < NW; w += 4) {
            const float4 x = *reinterpret_cast<const float4*>(ssm + t * NW + w);
            ss += (x.x + x.y) + (x.z + x.w);
          }
          inv = rsqrtf(ss * inv_dv + p.eps);
        }
        if (t < s0 || t >= s1) continue;
        const bf16* gr = gs + t * L::VCP;
        bf16* orow = reinterpret_cast<bf16*>(sp.fused_out) + (int64_t)(row0 + t0 + t) * sp.out_ld + (int64_t)h * p.dv;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int c = warp * 16 + j * 8 + (lane & 3) * 2;
          if (c >= p.dv) continue;
          float y[2] = {o[j][u * 2] * inv, o[j][u * 2 + 1] * inv};
          if (p.norm_w != nullptr) {
            y[0] *= __bfloat162float(p.norm_w[c]);
            if (c + 1 < p.dv) y[1] *= __bfloat162float(p.norm_w[c + 1]);
          }
          if (p.g != nullptr) {
            const float2 gg = unpack2(*reinterpret_cast<const uint32_t*>(gr + c));
            y[0] *= silu_fast(gg.x);
            y[1] *= silu_fast(gg.y);
          }
          if (p.vec_ok && c + 1 < p.dv) {
            *reinterpret_cast<bf162*>(orow + c) = __floats2bfloat162_rn(y[0], y[1]);
          } else {
            if (c < p.dv) orow[c] = __float2bfloat16(y[0]);
            if (c + 1 < p.dv) orow[c + 1] = __float2bfloat16(y[1]);
          }
        }
      }
    }
  }
  if (!STATE_ONLY && !one_seg) return;      // the scan has written the state behind the last segment
  __syncthreads();
  if (STATE_ONLY && c0 == 0)
    for (int c = tid; c < dk; c += NT) sp.decay[seg_at * dk + c] = exp2f(tot[c]);
  if (has_cols) {
#pragma unroll
    for (int nt = 0; nt < DK / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = nt * 8 + (lane & 3) * 2 + (e & 1), v = vrow + (e >> 1) * 8;
        if (c < dk && v < p.dv_pad) S[(int64_t)c * p.dv_pad + v] = acc[nt][e] * et[c];
      }
  }
}

// Segment states -> start states: S <- decay * S + local, from the slot's state (or zero) through the segments of a
// sequence; the state behind the last one goes to the slot.  grid (heads, sequences, parts of the dk x dv_pad matrix).
__global__ void __launch_bounds__(256) linattn_scan_kernel(LinAttnParams<bf16> p, SegParams sp) {
  const int h = blockIdx.x, b = blockIdx.y;
  const int i = (blockIdx.z * 256 + threadIdx.x) * 4;
  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q[b], n = p.cu_q[b + 1] - row0;
  const int slot = p.slots[b];
  if (n <= 0 || slot < 0 || i >= p.dk * p.dv_pad) return;
  const int c = i / p.dv_pad;
  float4* S = reinterpret_cast<float4*>(p.state + ((int64_t)slot * p.H + h) * p.dk * p.dv_pad + i);
  float4 s = p.kv_lens[b] == n ? make_float4(0.f, 0.f, 0.f, 0.f) : *S;
  const int segs = (n + sp.len - 1) / sp.len;
  for (int g = 0; g < segs; ++g) {
    const int64_t at = seg_slot(row0, b, g, sp.len) * p.H + h;
    float4* L = reinterpret_cast<float4*>(sp.state + at * p.dk * p.dv_pad + i);
    const float4 l = *L;
    const float d = sp.decay[at * p.dk + c];
    *L = s;
    s.x = d * s.x + l.x; s.y = d * s.y + l.y; s.z = d * s.z + l.z; s.w = d * s.w + l.w;
  }
  *S = s;
}

template <int DK, int NW, bool STATE_ONLY>
static int launch_chunk_kernel(const LinAttnParams<bf16>& p, const SegParams& sp, int segs, cudaStream_t s) {
  using L = ChunkSmem<DK, NW>;
  const int rot = p.cos_sin != nullptr ? p.rot : 0;
  const int RP = p.log_decay == nullptr ? (p.rank + 15) & ~15 : 0;
  const size_t smem = L::dyn + (size_t)2 * kLC * rot * 4 +
                      (RP ? (size_t)(kLC + 1) * DK * 4 + (size_t)2 * kLC * RP * 2 + (size_t)DK * (RP + 8) * 2 : 0);
  if (smem > 224 * 1024) return (int)cudaErrorInvalidValue;
  const cudaError_t e = cudaFuncSetAttribute(linattn_chunk_kernel<DK, NW, STATE_ONLY>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const int slices = (p.dv + L::VC - 1) / L::VC;
  launch_pdl(linattn_chunk_kernel<DK, NW, STATE_ONLY>, dim3(p.H, p.n_seqs, slices * segs), dim3(NW * 32), smem, s, p, sp);
  return XLLM_LAUNCH_CHECK();
}

template <int DK, int NW>
static int launch_chunk(const LinAttnParams<bf16>& p, SegParams sp, int segs, cudaStream_t s) {
  if (p.dv > NW * 16) sp.fused_out = nullptr;
  if (segs > 1) {
    int rc = launch_chunk_kernel<DK, NW, true>(p, sp, segs, s);
    if (rc != 0) return rc;
    const int n = p.dk * p.dv_pad;
    launch_pdl(linattn_scan_kernel, dim3(p.H, p.n_seqs, (n + 1023) / 1024), dim3(256), 0, s, p, sp);
    rc = XLLM_LAUNCH_CHECK();
    if (rc != 0) return rc;
  } else {
    sp.state = nullptr;
  }
  return launch_chunk_kernel<DK, NW, false>(p, sp, segs, s);
}

}  // namespace xllm

// Common arguments of the entry points below.  dtype: 0 bf16, 1 fp32.
//   state [slots, H, dk, dv_pad] fp32, dv_pad = dv rounded up to 4;  slots, kv_lens int32 [n_seqs]
//   q, k, v, g, r: column blocks of rows with stride ld (g, r may be null);  cos_sin null or [max_pos, rot]
//   log_decay fp32 [H], or null with a2 [H dk, rank], a2_b [H dk] and inv_tau
XLLM_API int xllm_linattn(void* state, const void* slots, const void* cu_q, const void* kv_lens, const void* q, const void* k,
                          const void* v, const void* g, const void* r, int64_t ld, const void* cos_sin, int64_t max_pos,
                          const void* positions, const void* log_decay, const void* a2, const void* a2_b, const void* norm_w,
                          void* out, int64_t out_ld, int n_seqs, int H, int dk, int dv, int rot, int interleaved, int rank,
                          int unit_norm, float q_scale, float k_scale, float inv_tau, float eps, int dtype, int mode,
                          void* seg_state, void* seg_decay, int seg_len, int segs, int finish, int in_silu, void* stream) {
  // in_silu: q, k and v pass through silu before anything else
  // mode 0: one token per sequence, sequence s is row s, `out` finished in the activation type, or without `finish` raw
  //         fp32 [rows, H, dv] (cu_q unused)
  // mode 1: prompt rows by cu_q, `out` raw fp32 [T, H, dv], or with `finish` (dv <= 128) finished bf16 rows [T, out_ld].
  //         Prompts longer than seg_len run as up to `segs` segments side by side: seg_state fp32 [n, H, dk, dv_pad] and
  //         seg_decay fp32 [n, H, dk] with n = T / seg_len + n_seqs + 1, seg_len a multiple of 16.
  // mode 2: prompt rows token by token, `out` raw fp32
  using namespace xllm;
  if (n_seqs == 0) return 0;
  if (H <= 0 || dk <= 0 || dv <= 0 || dk > 512 || dv > 1024 || rot < 0 || rot > dk || rot % 2 != 0)
    return (int)cudaErrorInvalidValue;
  if (log_decay == nullptr && (a2 == nullptr || a2_b == nullptr || r == nullptr || rank <= 0)) return (int)cudaErrorInvalidValue;
  if (mode != 0 && cu_q == nullptr) return (int)cudaErrorInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  int rc = 0;
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    LinAttnParams<T> p;
    p.state = (float*)state; p.slots = (const int32_t*)slots; p.cu_q = (const int32_t*)cu_q; p.kv_lens = (const int32_t*)kv_lens;
    p.q = (const T*)q; p.k = (const T*)k; p.v = (const T*)v; p.g = (const T*)g; p.r = (const T*)r; p.ld = ld;
    p.cos_sin = rot > 0 ? (const float*)cos_sin : nullptr; p.positions = (const int64_t*)positions; p.max_pos = max_pos;
    p.log_decay = (const float*)log_decay; p.a2 = (const T*)a2; p.a2_b = (const T*)a2_b; p.norm_w = (const T*)norm_w;
    p.out = out; p.out_ld = out_ld; p.n_seqs = n_seqs; p.H = H; p.dk = dk; p.dv = dv; p.dv_pad = (dv + 3) & ~3; p.rot = rot;
    p.interleaved = interleaved; p.rank = log_decay ? 0 : rank; p.unit_norm = unit_norm; p.q_scale = q_scale;
    p.k_scale = k_scale; p.inv_tau = inv_tau; p.eps = eps;
    p.in_silu = in_silu; p.raw_out = mode == 0 && !finish;
    const auto a16 = [](const void* x) { return (((uintptr_t)x) & 15) == 0; };
    p.vec_ok = dk % 8 == 0 && dv % 8 == 0 && ld % 8 == 0 && a16(q) && a16(k) && a16(v) &&
               (log_decay != nullptr || (rank % 8 == 0 && a16(r)));
    if (mode == 0) {
      const int CG = p.dv_pad >> 2, RG = 256 / CG;
      const size_t smem = (size_t)(3 * ((dk + 3) & ~3) + p.dv_pad + RG * p.dv_pad) * 4;
      const int rows = (dk + RG - 1) / RG;
      const dim3 grid(H, n_seqs), block(256);
      if (rows <= 4) launch_pdl(linattn_decode_kernel<T, 4>, grid, block, smem, s, p);
      else if (rows <= 8) launch_pdl(linattn_decode_kernel<T, 8>, grid, block, smem, s, p);
      else launch_pdl(linattn_decode_kernel<T, 16>, grid, block, smem, s, p);
      rc = XLLM_LAUNCH_CHECK();
      return;
    }
    if constexpr (sizeof(T) == 2) {
      if (mode == 1) {
        SegParams sp;
        sp.state = (float*)seg_state; sp.decay = (float*)seg_decay; sp.len = seg_len; sp.out_ld = out_ld;
        sp.fused_out = finish ? out : nullptr;
        if (finish) p.vec_ok = p.vec_ok && (g == nullptr || a16(g)) && out_ld % 2 == 0;
        if (seg_len <= 0 || seg_len % kLC != 0 || segs < 1 || (segs > 1 && (seg_state == nullptr || seg_decay == nullptr)) ||
            (finish && dv > 128)) {
          rc = (int)cudaErrorInvalidValue;
          return;
        }
        const bool wide = dv > 64;
        if (dk <= 64) rc = wide ? launch_chunk<64, 8>(p, sp, segs, s) : launch_chunk<64, 4>(p, sp, segs, s);
        else if (dk <= 128) rc = wide ? launch_chunk<128, 8>(p, sp, segs, s) : launch_chunk<128, 4>(p, sp, segs, s);
        else if (dk <= 256) rc = wide ? launch_chunk<256, 8>(p, sp, segs, s) : launch_chunk<256, 4>(p, sp, segs, s);
        else rc = (int)cudaErrorInvalidValue;
        return;
      }
    }
    const dim3 grid(H, n_seqs, (dv + 31) / 32), block(256);
    const size_t smem = (size_t)6 * dk * 4;
    if (dk <= 64) launch_pdl(linattn_recurrent_kernel<T, 2>, grid, block, smem, s, p);
    else if (dk <= 128) launch_pdl(linattn_recurrent_kernel<T, 4>, grid, block, smem, s, p);
    else if (dk <= 256) launch_pdl(linattn_recurrent_kernel<T, 8>, grid, block, smem, s, p);
    else launch_pdl(linattn_recurrent_kernel<T, 16>, grid, block, smem, s, p);
    rc = XLLM_LAUNCH_CHECK();
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return rc;
}
