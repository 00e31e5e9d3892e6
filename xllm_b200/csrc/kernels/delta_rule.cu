// Gated delta rule with one decay per head and KEY CHANNEL, per head:
//
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          S [dk, dv] fp32, one per state slot
//
// q, k and v pass a short causal convolution with silu; q and k are unit vectors per head (q scaled); heads may share
// q and k (heads / kv_heads neighbours).  g = exp(-exp(A_log) softplus(W_2 r + dt_bias)) with r a low-rank column block
// of the projection row; beta = sigmoid of an fp32 projection.  The output of a head is divided by its root mean square,
// weighted, and multiplied by the sigmoid of a gate.  The sibling of gdn.cu, whose decay is one number per head and
// whose inputs are prepared by tensor operations.
//
//   delta_decode_kernel        one token per sequence, from the projection rows and the decays to the finished row; the
//                              state crosses HBM once in each direction
//   conv_heads_kernel          prompts: convolution, silu, unit norm of q and k -> fp32
//   conv_ring_kernel           prompts: the last inputs of every sequence -> its ring
//   channel_decay_kernel       the decays, W_2 r on the tensor cores
//   delta_prefill_kernel       prompts: the recurrence, token by token with the state in registers (recurrence.cuh)
// (head_norm.cu finishes the prompts' rows.)
//
// A sequence whose rows in the batch are its first tokens (kv_len == number of rows) starts from S = 0 whatever its
// slot holds; slot < 0 marks padding rows.  Built without fast-math: errors of a decay multiply up over a sequence.
#include "attn_common.cuh"
#include "recurrence.cuh"
#include "short_conv.cuh"

namespace xllm {

template <typename T>
struct DeltaParams {
  float* state;              // [slots, H, dk, dv_pad]
  T* ring;                   // [slots, taps, C], C = 2 G dk + H dv: q | k | v channels
  const int32_t *slots, *cu_q, *kv_lens;
  const T *q, *k, *v, *r;    // column blocks of the projection rows
  int64_t ld;
  const float* zb;           // [rows, zb_ld] fp32: pre-sigmoid beta of head h in column h
  int64_t zb_ld;
  const T* conv_w;           // [C, taps]
  const T* a2;               // [H dk, rank]
  const T* dt_bias;          // [H dk]
  const T* a_log;            // [H]
  const T* gate;             // [rows, gate_ld] (decode)
  int64_t gate_ld;
  const T* norm_w;           // [dv]
  T* out;                    // [rows, out_ld] (decode)
  int64_t out_ld;
  float *qn, *kn;            // [rows, G, dkp] (prompts)
  float* vn;                 // [rows, H, dvp]
  float* gn;                 // [rows, H, dkp]
  float* o;                  // [rows, H, dv]
  int n_seqs, rows, row0, H, G, dk, dv, dkp, dvp, taps, rank;
  float q_scale, eps;
  __host__ __device__ int64_t channels() const { return (int64_t)2 * G * dk + (int64_t)H * dv; }
};

__device__ __forceinline__ float softplus_exact(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

constexpr float kUnitEps = 1e-6f;

// ------------------------------------------------------------------------------------------------ decode
// grid (heads, sequences), 256 threads: dvp / 4 column groups x row groups, NR rows of four columns per thread.
template <typename T, int NR>
__global__ void __launch_bounds__(256) delta_decode_kernel(DeltaParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  const int dk = p.dk, dv = p.dv, dvp = p.dvp, dkp = p.dkp;
  float* qs = sm;
  float* ks = qs + dkp;
  float* gs = ks + dkp;
  float* vs = gs + dkp;                    // [dvp]
  float* red = vs + dvp;                   // [RG][dvp]
  __shared__ float red32[2][32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
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
  float* S = p.state + (((int64_t)slot * p.H + h) * dk) * dvp + cg * 4;
  float4 s[NR];
#pragma unroll
  for (int u = 0; u < NR; ++u) {
    const int r = rg + u * RG;
    s[u] = (active && !fresh && r < dk) ? *reinterpret_cast<const float4*>(S + (int64_t)r * dvp)
                                        : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int pos = len - 1, g = h / (p.H / p.G), G = p.G, taps = p.taps;
  const int64_t C = p.channels();
  T* ring = p.ring + (int64_t)slot * taps * C;
  T* ring_now = ring + (int64_t)(pos % taps) * C;
  const bool keeps_qk = h % (p.H / G) == 0;
  // channels of this head in the order q | k | v; the token's own inputs go to its ring row
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < 2 * dk + dv; i += 256) {
    const T* x;
    int64_t c;
    if (i < dk) { x = p.q + b * p.ld + (int64_t)g * dk + i; c = (int64_t)g * dk + i; }
    else if (i < 2 * dk) { x = p.k + b * p.ld + (int64_t)g * dk + i - dk; c = (int64_t)(G + g) * dk + i - dk; }
    else { x = p.v + b * p.ld + (int64_t)h * dv + i - 2 * dk; c = (int64_t)2 * G * dk + (int64_t)h * dv + i - 2 * dk; }
    float y;
    conv_silu<T, 1>(x, p.ld, 0, pos, ring + c, C, p.conv_w + c * taps, taps, &y);
    if (i < dk) { qs[i] = y; sq += y * y; }
    else if (i < 2 * dk) { ks[i - dk] = y; sk += y * y; }
    else vs[i - 2 * dk] = y;
    if (taps > 1 && (keeps_qk || i >= 2 * dk)) ring_now[c] = *x;
  }
  for (int i = dv + tid; i < dvp; i += 256) vs[i] = 0.f;
  for (int i = tid; i < dk; i += 256) gs[i] = p.gn[((int64_t)b * p.H + h) * dkp + i];
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { red32[0][warp] = sq; red32[1][warp] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) { sq += red32[0][w]; sk += red32[1][w]; }
  const float iq = p.q_scale / sqrtf(sq + kUnitEps), ik = 1.f / sqrtf(sk + kUnitEps);
  for (int i = tid; i < dk; i += 256) {
    qs[i] *= iq;
    ks[i] *= ik;
  }
  const float beta = sigmoid_exact(p.zb[b * p.zb_ld + h]);
  __syncthreads();
  float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
#pragma unroll
    for (int u = 0; u < NR; ++u) {
      const int r = rg + u * RG;
      if (r >= dk) break;
      const float gg = gs[r], kk = ks[r];
      s[u].x *= gg; s[u].y *= gg; s[u].z *= gg; s[u].w *= gg;
      d.x += s[u].x * kk; d.y += s[u].y * kk; d.z += s[u].z * kk; d.w += s[u].w * kk;
    }
    *reinterpret_cast<float4*>(red + rg * dvp + cg * 4) = d;
  }
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    d = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int w = 0; w < RG; ++w) {
      const float4 x = *reinterpret_cast<const float4*>(red + w * dvp + cg * 4);
      d.x += x.x; d.y += x.y; d.z += x.z; d.w += x.w;
    }
    const float4 v4 = *reinterpret_cast<const float4*>(vs + cg * 4);
    const float4 w = make_float4(beta * (v4.x - d.x), beta * (v4.y - d.y), beta * (v4.z - d.z), beta * (v4.w - d.w));
#pragma unroll
    for (int u = 0; u < NR; ++u) {
      const int r = rg + u * RG;
      if (r >= dk) break;
      const float kk = ks[r], qq = qs[r];
      float4 x = s[u];
      x.x += kk * w.x; x.y += kk * w.y; x.z += kk * w.z; x.w += kk * w.w;
      *reinterpret_cast<float4*>(S + (int64_t)r * dvp) = x;
      o.x += qq * x.x; o.y += qq * x.y; o.z += qq * x.z; o.w += qq * x.w;
    }
  }
  __syncthreads();
  if (active) *reinterpret_cast<float4*>(red + rg * dvp + cg * 4) = o;
  __syncthreads();
  float ss = 0.f, mine = 0.f;              // dv <= 128: one element per thread
  if (tid < dv) {
    for (int w = 0; w < RG; ++w) mine += red[w * dvp + tid];
    ss = mine * mine;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red32[0]) / (float)dv + p.eps);
  if (tid < dv)
    orow[tid] = from_f32<T>(mine * inv * to_f32(p.norm_w[tid]) *
                            sigmoid_exact(to_f32(p.gate[b * p.gate_ld + (int64_t)h * dv + tid])));
}

// ------------------------------------------------------------------------------------------------ prompts: inputs
// one warp per (row, head of q | k | v); a lane owns V neighbouring channels out of every 32 V
template <typename T, int V>
__global__ void __launch_bounds__(256) conv_heads_kernel(DeltaParams<T> p) {
  constexpr int NI = V == 4 ? 4 : 16;
  const int lane = threadIdx.x & 31, items = 2 * p.G + p.H;
  const int64_t n = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  pdl_wait();
  pdl_launch_dependents();
  if (n >= (int64_t)(p.rows - p.row0) * items) return;
  const int row = p.row0 + (int)(n / items);
  int h = (int)(n - (int64_t)(row - p.row0) * items);
  const int b = seq_of_row(p.cu_q, p.n_seqs, row);
  if (b < 0 || p.slots[b] < 0) return;
  const int back = row - p.cu_q[b], pos = p.kv_lens[b] - (p.cu_q[b + 1] - row);
  const int part = h < p.G ? 0 : (h < 2 * p.G ? 1 : 2);
  h -= part == 0 ? 0 : (part == 1 ? p.G : 2 * p.G);
  const int d = part == 2 ? p.dv : p.dk, dp = part == 2 ? p.dvp : p.dkp;
  const int64_t c0 = (part == 2 ? (int64_t)2 * p.G * p.dk : (int64_t)part * p.G * p.dk) + (int64_t)h * d;
  const T* x = (part == 0 ? p.q : (part == 1 ? p.k : p.v)) + row * p.ld + (int64_t)h * d;
  const int64_t C = p.channels();
  const T* ring = p.ring + (int64_t)p.slots[b] * p.taps * C + c0;
  const T* w = p.conv_w + c0 * p.taps;
  float* dst = (part == 0 ? p.qn : (part == 1 ? p.kn : p.vn)) + ((int64_t)row * (part == 2 ? p.H : p.G) + h) * dp;
  float y[NI][V];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (lane + 32 * i) * V;
#pragma unroll
    for (int j = 0; j < V; ++j) y[i][j] = 0.f;
    if (c >= d) continue;
    conv_silu<T, V>(x + c, p.ld, back, pos, ring + c, C, w + (int64_t)c * p.taps, p.taps, y[i]);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += y[i][j] * y[i][j];
  }
  float f = 1.f;
  if (part < 2) f = (part == 0 ? p.q_scale : 1.f) / sqrtf(warp_sum(ss) + kUnitEps);
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (lane + 32 * i) * V;
    if (c >= dp) continue;                 // the padding behind d is written as zero
#pragma unroll
    for (int j = 0; j < V; ++j) y[i][j] *= f;
    store_f32<V>(dst + c, y[i]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) conv_ring_kernel(DeltaParams<T> p) {
  const int b = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, slot = p.slots[b];
  const int64_t c = (int64_t)blockIdx.x * 256 + threadIdx.x, C = p.channels();
  if (n <= 0 || slot < 0 || c >= C) return;
  const int64_t qk = (int64_t)p.G * p.dk;
  const T* x = c < qk ? p.q + c : (c < 2 * qk ? p.k + c - qk : p.v + c - 2 * qk);
  for (int i = max(0, n - (p.taps - 1)); i < n; ++i) {
    const int pos = p.kv_lens[b] - n + i;
    p.ring[((int64_t)slot * p.taps + pos % p.taps) * C + c] = x[(int64_t)(first + i) * p.ld];
  }
}

// 64 rows x 64 channels per CTA, four warps of 16 rows; z = W_2 r accumulates in fp32 from bf16 operands
__global__ void __launch_bounds__(128) channel_decay_tile_kernel(DeltaParams<bf16> p) {
  extern __shared__ __align__(16) uint8_t raw[];
  const int RP = (p.rank + 15) & ~15, st = RP + 8;
  bf16* rs = reinterpret_cast<bf16*>(raw);          // [64][st]
  bf16* ws = rs + 64 * st;                          // [64][st]
  const int r0 = p.row0 + blockIdx.x * 64, c0 = blockIdx.y * 64, tid = threadIdx.x, nc = p.H * p.dk;
  const int warp = tid >> 5, lane = tid & 31;
  const bf16 zero = __float2bfloat16(0.f);
  const bool v8 = p.rank % 8 == 0 && p.ld % 8 == 0 && (((uintptr_t)p.a2 | (uintptr_t)p.r) & 15) == 0;
  const uint4 zero8 = make_uint4(0, 0, 0, 0);
  const auto copy = [&](bf16* dst, const bf16* src, int64_t ld, int n) {     // n rows of `rank` elements, zeros behind
    if (v8) {
      const int per = RP >> 3;
      for (int i = tid; i < 64 * per; i += 128) {
        const int y = i / per, x = (i - y * per) * 8;
        *reinterpret_cast<uint4*>(dst + y * st + x) = (y < n && x < p.rank) ? *reinterpret_cast<const uint4*>(src + y * ld + x) : zero8;
      }
    } else {
      for (int i = tid; i < 64 * RP; i += 128) {
        const int y = i / RP, x = i - y * RP;
        dst[y * st + x] = (y < n && x < p.rank) ? src[y * ld + x] : zero;
      }
    }
  };
  copy(ws, p.a2 + (int64_t)c0 * p.rank, p.rank, nc - c0);
  pdl_wait();
  pdl_launch_dependents();
  copy(rs, p.r + (int64_t)r0 * p.ld, p.ld, p.rows - r0);
  __syncthreads();
  float z[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) z[n][e] = 0.f;
  const int ra = warp * 16 + (lane >> 2), kc = (lane & 3) * 2;
  for (int k = 0; k < RP; k += 16) {
    uint32_t a[4];
    a[0] = *reinterpret_cast<const uint32_t*>(rs + ra * st + k + kc);
    a[1] = *reinterpret_cast<const uint32_t*>(rs + (ra + 8) * st + k + kc);
    a[2] = *reinterpret_cast<const uint32_t*>(rs + ra * st + k + kc + 8);
    a[3] = *reinterpret_cast<const uint32_t*>(rs + (ra + 8) * st + k + kc + 8);
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const bf16* w = ws + (n * 8 + (lane >> 2)) * st + k + kc;
      mma_bf16_16816(z[n], a, *reinterpret_cast<const uint32_t*>(w), *reinterpret_cast<const uint32_t*>(w + 8));
    }
  }
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    const int c = c0 + n * 8 + kc;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      if (c + e >= nc) break;
      const int h = (c + e) / p.dk, ch = c + e - h * p.dk;
      const float A = expf(__bfloat162float(p.a_log[h])), bias = __bfloat162float(p.dt_bias[c + e]);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int row = r0 + ra + 8 * u;
        if (row < p.rows) p.gn[((int64_t)row * p.H + h) * p.dkp + ch] = expf(-A * softplus_exact(z[n][2 * u + e] + bias));
      }
    }
  }
}

// any type and rank: a thread per (row, channel)
template <typename T>
__global__ void __launch_bounds__(256) channel_decay_kernel(DeltaParams<T> p) {
  pdl_wait();
  pdl_launch_dependents();
  const int nc = p.H * p.dk;
  const int64_t total = (int64_t)(p.rows - p.row0) * nc;
  for (int64_t i = blockIdx.x * (int64_t)256 + threadIdx.x; i < total; i += (int64_t)gridDim.x * 256) {
    const int row = p.row0 + (int)(i / nc), c = (int)(i % nc), h = c / p.dk;
    float z = to_f32(p.dt_bias[c]);
    const T* r = p.r + (int64_t)row * p.ld;
    const T* w = p.a2 + (int64_t)c * p.rank;
    for (int j = 0; j < p.rank; ++j) z += to_f32(r[j]) * to_f32(w[j]);
    p.gn[((int64_t)row * p.H + h) * p.dkp + c - h * p.dk] = expf(-expf(to_f32(p.a_log[h])) * softplus_exact(z));
  }
}

// ------------------------------------------------------------------------------------------------ prompts: recurrence
// grid (slices of eight columns per warp, heads, sequences); the tile of the next tokens is fetched while one is worked on
struct DeltaScan {
  float* state;
  const int32_t *slots, *cu_q, *kv_lens;
  const float *qn, *kn, *vn, *gn, *zb;
  int64_t zb_ld;
  float* o;
  int H, G, dk, dv, dkp, dvp;
};

template <int J>
__global__ void __launch_bounds__(256) delta_prefill_kernel(DeltaScan p) {
  constexpr int DK = 32 * J, TT = kRecTile, UNROLL = J > 8 ? 1 : 2;
  extern __shared__ __align__(16) float sm[];
  const int cols = (blockDim.x >> 5) * kRecCols;                 // of this CTA
  const int stage = TT * (3 * DK + cols) + TT;                   // floats of a stage: q | k | g | v | beta
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rgrp = lane & 7, c0 = blockIdx.x * cols, lc = warp * kRecCols + (lane >> 3) * 2, col = c0 + lc;
  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q[b], n = p.cu_q[b + 1] - row0, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;
  float* S = p.state + (((int64_t)slot * p.H + h) * p.dk) * p.dvp + col;
  StateColumns<J> st;
  st.load(S, p.dk, p.dvp, rgrp, col < p.dvp && p.kv_lens[b] != n);
  const int g = h / (p.H / p.G), kv4 = p.dkp >> 2, v4 = cols >> 2;
  for (int i = tid; i < 2 * stage; i += blockDim.x) sm[i] = 0.f;  // what lies behind dk and dv stays zero
  __syncthreads();
  const auto fetch = [&](int t0, int buf) {
    float* base = sm + buf * stage;
    const int m = min(TT, n - t0);
    for (int i = tid; i < m * kv4; i += blockDim.x) {
      const int t = i / kv4, c = (i - t * kv4) * 4;
      const int64_t row = row0 + t0 + t, qk = (row * p.G + g) * p.dkp + c;
      cp_async16(smem_u32(base + t * DK + c), p.qn + qk, true);
      cp_async16(smem_u32(base + (TT + t) * DK + c), p.kn + qk, true);
      cp_async16(smem_u32(base + (2 * TT + t) * DK + c), p.gn + (row * p.H + h) * p.dkp + c, true);
    }
    for (int i = tid; i < m * v4; i += blockDim.x) {
      const int t = i / v4, c = (i - t * v4) * 4;
      if (c0 + c < p.dvp)
        cp_async16(smem_u32(base + 3 * TT * DK + t * cols + c), p.vn + ((int64_t)(row0 + t0 + t) * p.H + h) * p.dvp + c0 + c, true);
    }
    if (tid < m) base[3 * TT * DK + TT * cols + tid] = sigmoid_exact(p.zb[(int64_t)(row0 + t0 + tid) * p.zb_ld + h]);
    cp_async_commit();
  };
  fetch(0, 0);
  int buf = 0;
  for (int t0 = 0; t0 < n; t0 += TT, buf ^= 1) {
    cp_async_wait<0>();
    __syncthreads();
    if (t0 + TT < n) fetch(t0 + TT, buf ^ 1);
    const float* base = sm + buf * stage;
    const float* vb = base + 3 * TT * DK + lc;
    const float* bb = base + 3 * TT * DK + TT * cols;
    const int m = min(TT, n - t0);
    float* orow = p.o + ((int64_t)(row0 + t0) * p.H + h) * p.dv + col + (lane & 1);
    const bool writes = rgrp < 2 && col + (lane & 1) < p.dv;
#pragma unroll UNROLL
    for (int t = 0; t < m; ++t) {
      f2 kf[2 * J], xf[2 * J];
      load_rows<J>(base + (2 * TT + t) * DK, rgrp, xf);           // decays
      load_rows<J>(base + (TT + t) * DK, rgrp, kf);
      f2 d0 = 0, d1 = 0, e0 = 0, e1 = 0;                          // packed zeros
#pragma unroll
      for (int j = 0; j < 2 * J; j += 2) {
        st.s[0][j] = mul_f2(st.s[0][j], xf[j]);
        st.s[1][j] = mul_f2(st.s[1][j], xf[j]);
        st.s[0][j + 1] = mul_f2(st.s[0][j + 1], xf[j + 1]);
        st.s[1][j + 1] = mul_f2(st.s[1][j + 1], xf[j + 1]);
        d0 = fma_f2(st.s[0][j], kf[j], d0);
        d1 = fma_f2(st.s[1][j], kf[j], d1);
        e0 = fma_f2(st.s[0][j + 1], kf[j + 1], e0);
        e1 = fma_f2(st.s[1][j + 1], kf[j + 1], e1);
      }
      const float2 a0 = unpack_f2(add_f2(d0, e0)), a1 = unpack_f2(add_f2(d1, e1));
      const float k0 = sum_row_groups(a0.x + a0.y), k1 = sum_row_groups(a1.x + a1.y);
      const float2 v = *reinterpret_cast<const float2*>(vb + t * cols);
      const float beta = bb[t];
      const float u0 = beta * (v.x - k0), u1 = beta * (v.y - k1);
      const f2 w0 = pack_f2(u0, u0), w1 = pack_f2(u1, u1);
      load_rows<J>(base + t * DK, rgrp, xf);                      // queries
      d0 = d1 = e0 = e1 = 0;
#pragma unroll
      for (int j = 0; j < 2 * J; j += 2) {
        st.s[0][j] = fma_f2(kf[j], w0, st.s[0][j]);
        st.s[1][j] = fma_f2(kf[j], w1, st.s[1][j]);
        st.s[0][j + 1] = fma_f2(kf[j + 1], w0, st.s[0][j + 1]);
        st.s[1][j + 1] = fma_f2(kf[j + 1], w1, st.s[1][j + 1]);
        d0 = fma_f2(st.s[0][j], xf[j], d0);
        d1 = fma_f2(st.s[1][j], xf[j], d1);
        e0 = fma_f2(st.s[0][j + 1], xf[j + 1], e0);
        e1 = fma_f2(st.s[1][j + 1], xf[j + 1], e1);
      }
      const float2 y0 = unpack_f2(add_f2(d0, e0)), y1 = unpack_f2(add_f2(d1, e1));
      const float y = sum_row_groups_2(y0.x + y0.y, y1.x + y1.y);
      if (writes) orow[(int64_t)t * p.H * p.dv] = y;
    }
  }
  if (col < p.dvp) st.store(S, p.dk, p.dvp, rgrp);
}

template <typename T>
static int launch_channel_decay(const DeltaParams<T>& p, cudaStream_t s) {
  const int n = p.rows - p.row0;
  if constexpr (sizeof(T) == 2) {
    if (p.rank <= 256) {
      const size_t smem = (size_t)2 * 64 * (((p.rank + 15) & ~15) + 8) * 2;
      const cudaError_t e = cudaFuncSetAttribute(channel_decay_tile_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
      launch_pdl(channel_decay_tile_kernel, dim3((n + 63) / 64, (p.H * p.dk + 63) / 64), dim3(128), smem, s, p);
      return XLLM_LAUNCH_CHECK();
    }
  }
  const int64_t blocks = ((int64_t)n * p.H * p.dk + 255) / 256;
  launch_pdl(channel_decay_kernel<T>, dim3((unsigned)(blocks < 148 * 16 ? blocks : 148 * 16)), dim3(256), 0, s, p);
  return XLLM_LAUNCH_CHECK();
}

template <int J>
static int launch_delta_prefill(const DeltaScan& p, int n_seqs, cudaStream_t s) {
  const int warps = min(8, (p.dvp + kRecCols - 1) / kRecCols), cols = warps * kRecCols;
  const size_t smem = (size_t)2 * (kRecTile * (3 * 32 * J + cols) + kRecTile) * 4;
  const cudaError_t e = cudaFuncSetAttribute(delta_prefill_kernel<J>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  launch_pdl(delta_prefill_kernel<J>, dim3((p.dvp + cols - 1) / cols, p.H, n_seqs), dim3(warps * 32), smem, s, p);
  return XLLM_LAUNCH_CHECK();
}

}  // namespace xllm

// dtype: 0 bf16, 1 fp32 (projection rows, weights, ring, finished rows).
//   state [slots, H, dk, dvp] fp32, dvp = dv rounded up to 4;  ring [slots, taps, 2 G dk + H dv]
//   q, k, v, r: column blocks of rows with stride ld;  zb fp32 [rows, zb_ld]
// gn [rows, H, dkp] fp32 is scratch (dkp = dk rounded up to 4, zeros behind dk).
// mode 0: one token per sequence (sequence s is row s): gate, norm_w, out are used; dk <= 256, dv <= 128
// mode 1: rows [row0, rows) by cu_q: qn, kn [rows, G, dkp], vn [rows, H, dvp] are scratch, the raw fp32 outputs go to o [rows, H, dv];  dk <= 512
XLLM_API int xllm_delta_rule(void* state, void* ring, const void* slots, const void* cu_q, const void* kv_lens, const void* q,
                             const void* k, const void* v, const void* r, int64_t ld, const void* zb, int64_t zb_ld,
                             const void* conv_w, const void* a2, const void* dt_bias, const void* a_log, const void* gate,
                             int64_t gate_ld, const void* norm_w, void* out, int64_t out_ld, void* qn, void* kn, void* vn,
                             void* gn, void* o, int n_seqs, int rows, int row0, int H, int G, int dk, int dv, int taps,
                             int rank, float q_scale, float eps, int dtype, int mode, void* stream) {
  using namespace xllm;
  if (n_seqs == 0 || rows - row0 <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || dk <= 0 || dk > 512 || dv <= 0 || taps <= 0 || rank <= 0)
    return (int)cudaErrorInvalidValue;
  if (mode == 0 && (dk > 256 || dv > 128)) return (int)cudaErrorInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  int rc = 0;
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    DeltaParams<T> p;
    p.state = (float*)state; p.ring = (T*)ring; p.slots = (const int32_t*)slots; p.cu_q = (const int32_t*)cu_q;
    p.kv_lens = (const int32_t*)kv_lens; p.q = (const T*)q; p.k = (const T*)k; p.v = (const T*)v; p.r = (const T*)r; p.ld = ld;
    p.zb = (const float*)zb; p.zb_ld = zb_ld; p.conv_w = (const T*)conv_w; p.a2 = (const T*)a2; p.dt_bias = (const T*)dt_bias;
    p.a_log = (const T*)a_log; p.gate = (const T*)gate; p.gate_ld = gate_ld; p.norm_w = (const T*)norm_w; p.out = (T*)out;
    p.out_ld = out_ld; p.qn = (float*)qn; p.kn = (float*)kn; p.vn = (float*)vn; p.gn = (float*)gn; p.o = (float*)o;
    p.n_seqs = n_seqs; p.rows = rows; p.row0 = row0; p.H = H; p.G = G; p.dk = dk; p.dv = dv; p.dkp = (dk + 3) & ~3;
    p.dvp = (dv + 3) & ~3; p.taps = taps; p.rank = rank; p.q_scale = q_scale; p.eps = eps;
    if ((rc = launch_channel_decay(p, s)) != 0) return;
    if (mode == 0) {
      const int RG = 256 / (p.dvp >> 2), nr = (dk + RG - 1) / RG;
      const size_t smem = (size_t)(3 * p.dkp + p.dvp + RG * p.dvp) * 4;
      const dim3 grid(H, n_seqs), block(256);
      if (nr <= 4) launch_pdl(delta_decode_kernel<T, 4>, grid, block, smem, s, p);
      else if (nr <= 8) launch_pdl(delta_decode_kernel<T, 8>, grid, block, smem, s, p);
      else if (nr <= 16) launch_pdl(delta_decode_kernel<T, 16>, grid, block, smem, s, p);
      else launch_pdl(delta_decode_kernel<T, 32>, grid, block, smem, s, p);
      rc = XLLM_LAUNCH_CHECK();
      return;
    }
    const auto al = [](const void* x, size_t a) { return (((uintptr_t)x) & (a - 1)) == 0; };
    const size_t va = 4 * sizeof(T);
    const bool v4 = dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && al(q, va) && al(k, va) && al(v, va) && al(ring, va);
    const int64_t warps = (int64_t)(rows - row0) * (2 * G + H);
    const dim3 grid((unsigned)((warps + 7) / 8));
    if (v4) launch_pdl(conv_heads_kernel<T, 4>, grid, dim3(256), 0, s, p);
    else launch_pdl(conv_heads_kernel<T, 1>, grid, dim3(256), 0, s, p);
    if ((rc = XLLM_LAUNCH_CHECK()) != 0) return;
    if (taps > 1) {
      launch_pdl(conv_ring_kernel<T>, dim3((unsigned)((p.channels() + 255) / 256), n_seqs), dim3(256), 0, s, p);
      if ((rc = XLLM_LAUNCH_CHECK()) != 0) return;
    }
    DeltaScan d{p.state, p.slots, p.cu_q, p.kv_lens, p.qn, p.kn, p.vn, p.gn, p.zb, zb_ld, p.o, H, G, dk, dv, p.dkp, p.dvp};
    if (dk <= 32) rc = launch_delta_prefill<1>(d, n_seqs, s);
    else if (dk <= 64) rc = launch_delta_prefill<2>(d, n_seqs, s);
    else if (dk <= 96) rc = launch_delta_prefill<3>(d, n_seqs, s);
    else if (dk <= 128) rc = launch_delta_prefill<4>(d, n_seqs, s);
    else if (dk <= 192) rc = launch_delta_prefill<6>(d, n_seqs, s);
    else if (dk <= 256) rc = launch_delta_prefill<8>(d, n_seqs, s);
    else rc = launch_delta_prefill<16>(d, n_seqs, s);
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return rc;
}
