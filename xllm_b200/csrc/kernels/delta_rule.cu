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
//   conv_heads_kernel          convolution, silu, unit norm of q and k -> fp32
//   delta_decode_kernel        one token per sequence, from there to the finished row; the state crosses HBM once in each
//                              direction
//   conv_ring_kernel           prompts: the last inputs of every sequence -> its ring
//   channel_decay_kernel       the decays, W_2 r on the tensor cores
//   delta_chunk_prep_kernel,   prompts, bf16: sixteen tokens at a time on the tensor cores (below)
//   delta_chunk_kernel
//   delta_prefill_kernel       prompts of any type and size: token by token in fp32 with the state in registers
//                              (recurrence.cuh)
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
  const T* conv_w;           // [taps, C], the last row is the current token's
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
  int write_ring;            // one row per sequence: its inputs go to the ring as they pass
  int log_decay;             // gn receives log2 of the decays (chunked prompts)
  __host__ __device__ int64_t channels() const { return (int64_t)2 * G * dk + (int64_t)H * dv; }
};

__device__ __forceinline__ float softplus_exact(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// log(1 + e) = 2 artanh(s), s = e / (2 + e) <= 1/3 for e <= 1: six terms of the series leave a relative error of 2e-7
__device__ __forceinline__ float softplus_series(float z) {
  const float e = __expf(-fabsf(z)), s = __fdividef(e, 2.f + e), q = s * s;
  const float y = 1.f + q * (1.f / 3 + q * (1.f / 5 + q * (1.f / 7 + q * (1.f / 9 + q * (1.f / 11)))));
  return fmaxf(z, 0.f) + 2.f * s * y;
}
// 2^x, flushing denormal results
__device__ __forceinline__ float exp2_flush(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

constexpr float kUnitEps = 1e-6f;

// ------------------------------------------------------------------------------------------------ decode
// grid (heads, sequences), 256 threads: dvp / 4 column groups x row groups, NR rows of four columns per thread.
template <typename T, int NR>
__global__ void __launch_bounds__(256, NR <= 8 ? 3 : (NR <= 16 ? 2 : 1)) delta_decode_kernel(DeltaParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  const int dk = p.dk, dv = p.dv, dvp = p.dvp, dkp = p.dkp;
  float* qs = sm;
  float* ks = qs + dkp;
  float* gs = ks + dkp;
  float* vs = gs + dkp;                    // [dvp]
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
  float* S = p.state + (((int64_t)slot * p.H + h) * dk) * dvp + cg * 4;
  float4 s[NR];
#pragma unroll
  for (int u = 0; u < NR; ++u) {
    const int r = rg + u * RG;
    s[u] = (active && !fresh && r < dk) ? *reinterpret_cast<const float4*>(S + r * dvp) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int64_t qk = ((int64_t)b * p.G + h / (p.H / p.G)) * dkp, row = (int64_t)b * p.H + h;
  for (int i = tid; i < dk; i += 256) {
    qs[i] = p.qn[qk + i];
    ks[i] = p.kn[qk + i];
    gs[i] = p.gn[row * dkp + i];
  }
  for (int i = tid; i < dvp; i += 256) vs[i] = p.vn[row * dvp + i];
  const float beta = sigmoid_exact(p.zb[b * p.zb_ld + h]);
  const float g_out = tid < dv ? to_f32(p.gate[b * p.gate_ld + (int64_t)h * dv + tid]) : 0.f;
  const float w_out = tid < dv ? to_f32(p.norm_w[tid]) : 0.f;
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
      *reinterpret_cast<float4*>(S + r * dvp) = x;
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
  const float inv = 1.f / sqrtf(block_sum(ss, red32) / (float)dv + p.eps);
  if (tid < dv) orow[tid] = from_f32<T>(mine * inv * w_out * sigmoid_as<T>(g_out));
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
  const T* w = p.conv_w + c0;
  float* dst = (part == 0 ? p.qn : (part == 1 ? p.kn : p.vn)) + ((int64_t)row * (part == 2 ? p.H : p.G) + h) * dp;
  float y[NI][V];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (lane + 32 * i) * V;
#pragma unroll
    for (int j = 0; j < V; ++j) y[i][j] = 0.f;
    if (c >= d) continue;
    conv_silu<T, V>(x + c, p.ld, back, pos, ring + c, C, w + c, p.taps, y[i]);
    if (p.write_ring) {
      T* now = p.ring + ((int64_t)p.slots[b] * p.taps + pos % p.taps) * C + c0 + c;
#pragma unroll
      for (int j = 0; j < V; ++j) now[j] = x[c + j];
    }
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

// The same for up to four taps and heads of up to 128 channels: one warp per (run of rows, head), which reads every input
// once and keeps the last ones in registers; a lane owns four neighbouring channels.
template <typename T, int RUN>
__global__ void __launch_bounds__(256, 4) conv_heads_run_kernel(DeltaParams<T> p) {
  const int lane = threadIdx.x & 31, items = 2 * p.G + p.H;
  const unsigned it = blockIdx.x * 8 + (threadIdx.x >> 5), run = it / items;
  pdl_wait();
  pdl_launch_dependents();
  const int first = p.row0 + (int)run * RUN;
  if (first >= p.rows) return;
  int h = (int)(it - run * items);
  const int part = h < p.G ? 0 : (h < 2 * p.G ? 1 : 2);
  h -= part == 0 ? 0 : (part == 1 ? p.G : 2 * p.G);
  const int d = part == 2 ? p.dv : p.dk, c = lane * 4;
  const int64_t c0 = (part == 2 ? (int64_t)2 * p.G * p.dk : (int64_t)part * p.G * p.dk) + (int64_t)h * d + c, C = p.channels();
  const T* x = (part == 0 ? p.q : (part == 1 ? p.k : p.v)) + (int64_t)h * d + c;
  float* dst = (part == 0 ? p.qn : (part == 1 ? p.kn : p.vn)) + (int64_t)h * d + c;
  const int64_t dst_ld = (int64_t)(part == 2 ? p.H : p.G) * d;      // d is a multiple of 4: no padding
  const bool on = c < d;
  float v[RUN + 3][4], w[4][4];                                // w[taps back][channel]
#pragma unroll
  for (int r = 0; r < RUN + 3; ++r) {
    const int row = first + r - 3;
#pragma unroll
    for (int j = 0; j < 4; ++j) v[r][j] = 0.f;
    if (on && row >= 0 && row < p.rows) load_f32<4>(x + row * p.ld, v[r]);
  }
#pragma unroll
  for (int b = 0; b < 4; ++b)
  {
#pragma unroll
    for (int j = 0; j < 4; ++j) w[b][j] = 0.f;
    if (on && b < p.taps) load_f32<4>(p.conv_w + (p.taps - 1 - b) * C + c0, w[b]);
  }
  int b = -1, begin = 0, end = 0;
#pragma unroll
  for (int r = 0; r < RUN; ++r) {
    const int row = first + r;
    if (row >= p.rows) break;
    if (row >= end) {                                               // the row starts another sequence, or is the first
      b = seq_of_row(p.cu_q, p.n_seqs, row);
      begin = b < 0 ? row : p.cu_q[b];
      end = b < 0 ? row + 1 : p.cu_q[b + 1];
    }
    const int slot = b < 0 ? -1 : p.slots[b];
    if (slot < 0) continue;
    const int back = row - begin;
    float y[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      y[j] = v[r + 3][j] * w[0][j];
      if (back >= 1) y[j] += v[r + 2][j] * w[1][j];
      if (back >= 2) y[j] += v[r + 1][j] * w[2][j];
      if (back >= 3) y[j] += v[r][j] * w[3][j];
    }
    if (back < p.taps - 1) {                                        // inputs of earlier steps
      const int pos = p.kv_lens[b] - (end - row), now = pos % p.taps;
      for (int t = back + 1; t < p.taps && t <= pos && on; ++t) {
        float z[4];
        load_f32<4>(p.ring + ((int64_t)slot * p.taps + now - t + (t > now ? p.taps : 0)) * C + c0, z);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] += z[j] * (t == 1 ? w[1][j] : (t == 2 ? w[2][j] : w[3][j]));
      }
    }
    if (p.write_ring && on)
      store_f32<4>(p.ring + ((int64_t)slot * p.taps + (p.kv_lens[b] - 1) % p.taps) * C + c0, v[r + 3]);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      y[j] = silu_as<T>(y[j]);
      ss += y[j] * y[j];
    }
    if (part < 2) {
      const float f = (part == 0 ? p.q_scale : 1.f) * rsqrtf(warp_sum(ss) + kUnitEps);
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] *= f;
    }
    if (on) store_f32<4>(dst + row * dst_ld, y);
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
  __shared__ float rate[64], bias[64];              // -exp(A_log), dt_bias
  __shared__ int64_t at[64];                        // column of the output row
  const int r0 = p.row0 + blockIdx.x * 64, c0 = blockIdx.y * 64, tid = threadIdx.x, nc = p.H * p.dk;
  const int warp = tid >> 5, lane = tid & 31;
  const bf16 zero = __float2bfloat16(0.f);
  const bool v8 = p.rank % 8 == 0 && p.ld % 8 == 0 && (((uintptr_t)p.a2 | (uintptr_t)p.r) & 15) == 0;
  const auto copy = [&](bf16* dst, const bf16* src, int64_t ld, int n) {     // n rows of `rank` elements, zeros behind
    if (v8) {
      const int per = RP >> 3;
      for (int i = tid; i < 64 * per; i += 128) {
        const int y = i / per, x = (i - y * per) * 8;
        const bool ok = y < n && x < p.rank;
        cp_async16(smem_u32(dst + y * st + x), ok ? src + y * ld + x : src, ok);
      }
    } else {
      for (int i = tid; i < 64 * RP; i += 128) {
        const int y = i / RP, x = i - y * RP;
        dst[y * st + x] = (y < n && x < p.rank) ? src[y * ld + x] : zero;
      }
    }
  };
  copy(ws, p.a2 + (int64_t)c0 * p.rank, p.rank, nc - c0);
  if (tid < 64 && c0 + tid < nc) {
    const int h = (c0 + tid) / p.dk;
    rate[tid] = -expf(__bfloat162float(p.a_log[h])) * (p.log_decay ? 1.44269504088896341f : 1.f);
    bias[tid] = __bfloat162float(p.dt_bias[c0 + tid]);
    at[tid] = (int64_t)h * p.dkp + c0 + tid - h * p.dk;
  }
  pdl_wait();
  pdl_launch_dependents();
  copy(rs, p.r + (int64_t)r0 * p.ld, p.ld, p.rows - r0);
  cp_async_commit();
  cp_async_wait<0>();
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
  const int64_t ld = (int64_t)p.H * p.dkp;
  const bool pairs = p.dkp == p.dk && p.dk % 2 == 0;         // a pair of channels is one 8-byte store
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    const int c = n * 8 + kc;
    if (c0 + c >= nc) break;
    const bool two = c0 + c + 1 < nc;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int row = r0 + ra + 8 * u;
      if (row >= p.rows) continue;
      float g0 = rate[c] * softplus_series(z[n][2 * u] + bias[c]);
      float g1 = two ? rate[c + 1] * softplus_series(z[n][2 * u + 1] + bias[c + 1]) : 0.f;
      if (!p.log_decay) { g0 = expf(g0); g1 = expf(g1); }
      float* dst = p.gn + row * ld;
      if (pairs) {
        *reinterpret_cast<float2*>(dst + at[c]) = make_float2(g0, g1);
      } else {
        dst[at[c]] = g0;
        if (two) dst[at[c + 1]] = g1;
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
    const float g = -expf(to_f32(p.a_log[h])) * softplus_exact(z);
    p.gn[((int64_t)row * p.H + h) * p.dkp + c - h * p.dk] = p.log_decay ? g * 1.44269504088896341f : expf(g);
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

// ------------------------------------------------------------------------------------------------ prompts, chunks of 16
// With L_t the log2 decay from a chunk's start through token t (per key channel), S_0 the state before the chunk and
//
//   A_ts = sum_c k_t k_s 2^(L_t - L_s)  (s < t),     P_ts = sum_c q_t k_s 2^(L_t - L_s)  (s <= t),
//   M = (I + diag(beta) A)^-1 diag(beta)
//
// the chunk is   U = M (V - (k 2^L) S_0),   O = (q 2^L) S_0 + P U,   S <- 2^(L_end) S_0 + (k 2^(L_end - L))^T U.
//
// Everything but S_0 and V is made by delta_chunk_prep_kernel, all chunks side by side, and stored as the operands the
// tensor cores read: k 2^L, q 2^L, k 2^(L_end - L), M and P, each fp32 value as two bf16 terms.  All their decays are at
// most 1.  A and P factor their decays against the chunk's middle token; channels whose decays span more than fp32 holds
// take their share pair by pair instead.  delta_chunk_kernel walks the chunks of a sequence: a warp owns 16 state columns
// for all of dk as fp32 accumulators of S^T, which are the A operand of S^T (k 2^L)^T and S^T (q 2^L)^T without leaving
// the registers, as U^T is of the products after it.
constexpr int kDC = 16;
constexpr int kDWarps = 4;                   // warps of 16 columns
constexpr int kDStages = 3;
constexpr float kDLogRange = 86.f;

template <int DK>
struct ChunkBlob {                           // bytes of one (chunk, head), in this order
  static constexpr int tile = kDC * DK * 2;  // [16][DK] bf16, 16-byte pieces swizzled
  static constexpr int kt = 0, qt = 2 * tile, kc = 4 * tile;      // first and second term behind one another
  static constexpr int m = 6 * tile, p = m + 2 * kDC * kDC * 2;   // [16][16] bf16, two terms
  static constexpr int end = p + 2 * kDC * kDC * 2;               // [DK] fp32: 2^(L_end)
  static constexpr int bytes = end + DK * 4;
};

// chunk i of sequence b: unique because a sequence of n rows has at most n / 16 + 1 chunks
__device__ __forceinline__ int64_t chunk_slot(int row0, int b, int i) { return (int64_t)row0 / kDC + b + i; }

struct DeltaChunk {
  DeltaScan s;
  uint8_t* blobs;                            // [chunk slots, H, ChunkBlob]
};

// grid (chunks of a sequence, heads, sequences), 256 threads; a warp owns every eighth group of 16 channels.
template <int DK>
__global__ void __launch_bounds__(256) delta_chunk_prep_kernel(DeltaChunk d) {
  using B = ChunkBlob<DK>;
  constexpr int CH = DK / 8;
  const DeltaScan& p = d.s;
  __shared__ float part[8][2][kDC][kDC + 1];
  __shared__ float am[kDC][kDC + 1];
  __shared__ float betas[kDC];
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_wait();
  pdl_launch_dependents();
  const int row_first = p.cu_q[b], n_seq = p.cu_q[b + 1] - row_first;
  const int i0 = blockIdx.x * kDC;
  if (i0 >= n_seq || p.slots[b] < 0) return;
  const int n = min(kDC, n_seq - i0), row0 = row_first + i0;
  uint8_t* blob = d.blobs + (chunk_slot(row_first, b, blockIdx.x) * p.H + h) * B::bytes;
  if (tid < kDC) betas[tid] = tid < n ? sigmoid_exact(p.zb[(int64_t)(row0 + tid) * p.zb_ld + h]) : 0.f;
  const int g = h / (p.H / p.G), ta = lane >> 2, kc = (lane & 3) * 2;
  float ca[2][4], cp[2][4];                  // A and P: rows ta (+ 8), columns 8 j + kc (+ 1)
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) ca[j][e] = cp[j][e] = 0.f;
  for (int c0 = warp * 16; c0 < DK; c0 += 128) {
    // elements [u][v]: token ta + 8 u, channels c0 + 8 v + kc, + 1
    float2 q[2][2], k[2][2], L[2][2];
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int v = 0; v < 2; ++v) {
        const int c = c0 + 8 * v + kc;
        const int64_t row = row0 + ta + 8 * u;
        q[u][v] = k[u][v] = L[u][v] = make_float2(0.f, 0.f);
        if (ta + 8 * u < n && c < p.dkp) {   // dkp is a multiple of 4, zeros behind dk
          const int64_t at = (row * p.G + g) * p.dkp + c;
          q[u][v] = *reinterpret_cast<const float2*>(p.qn + at);
          k[u][v] = *reinterpret_cast<const float2*>(p.kn + at);
          L[u][v] = *reinterpret_cast<const float2*>(p.gn + (row * p.H + h) * p.dkp + c);
        }
      }
    float2 ref[2], end[2];
    bool unsafe = false;
#pragma unroll
    for (int v = 0; v < 2; ++v) {
#pragma unroll
      for (int s = 4; s < 32; s <<= 1) {
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const float x = __shfl_up_sync(0xffffffffu, L[u][v].x, s), y = __shfl_up_sync(0xffffffffu, L[u][v].y, s);
          if (lane >= s) { L[u][v].x += x; L[u][v].y += y; }
        }
      }
      ref[v].x = __shfl_sync(0xffffffffu, L[0][v].x, 28 + (lane & 3));     // token 7
      ref[v].y = __shfl_sync(0xffffffffu, L[0][v].y, 28 + (lane & 3));
      L[1][v].x += ref[v].x;
      L[1][v].y += ref[v].y;
      end[v].x = __shfl_sync(0xffffffffu, L[1][v].x, 28 + (lane & 3));     // rows behind the last one add nothing
      end[v].y = __shfl_sync(0xffffffffu, L[1][v].y, 28 + (lane & 3));
#pragma unroll
      for (int u = 0; u < 2; ++u)
        unsafe |= fabsf(L[u][v].x - ref[v].x) > kDLogRange || fabsf(L[u][v].y - ref[v].y) > kDLogRange;
    }
    if (lane < 4) {
#pragma unroll
      for (int v = 0; v < 2; ++v)
        *reinterpret_cast<float2*>(blob + B::end + (c0 + 8 * v + kc) * 4) = make_float2(exp2_flush(end[v].x), exp2_flush(end[v].y));
    }
    uint32_t hi, lo;
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int v = 0; v < 2; ++v) {
        const uint32_t at = swz<CH>(ta + 8 * u, (c0 >> 3) + v) + kc * 2;
        const auto put = [&](int where, float x, float y) {
          split_pack(x, y, hi, lo);
          *reinterpret_cast<uint32_t*>(blob + where + at) = hi;
          *reinterpret_cast<uint32_t*>(blob + where + B::tile + at) = lo;
        };
        const float ex = exp2_flush(L[u][v].x), ey = exp2_flush(L[u][v].y);
        put(B::kt, k[u][v].x * ex, k[u][v].y * ey);
        put(B::qt, q[u][v].x * ex, q[u][v].y * ey);
        put(B::kc, k[u][v].x * exp2_flush(end[v].x - L[u][v].x), k[u][v].y * exp2_flush(end[v].y - L[u][v].y));
      }
    if (!__any_sync(0xffffffffu, unsafe)) {
      uint32_t kh[4], kl[4], qh[4], ql[4], sh[4], sl[4];     // [2 v + u]: A fragments; s: B fragments [2 v + token half]
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int v = 0; v < 2; ++v) {
          const float dx = L[u][v].x - ref[v].x, dy = L[u][v].y - ref[v].y;
          const float ex = exp2_flush(dx), ey = exp2_flush(dy);
          split_pack(k[u][v].x * ex, k[u][v].y * ey, kh[2 * v + u], kl[2 * v + u]);
          split_pack(q[u][v].x * ex, q[u][v].y * ey, qh[2 * v + u], ql[2 * v + u]);
          split_pack(k[u][v].x * exp2_flush(-dx), k[u][v].y * exp2_flush(-dy), sh[2 * v + u], sl[2 * v + u]);
        }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma_bf16_16816(ca[j], kh, sh[j], sh[2 + j]);
        mma_bf16_16816(cp[j], qh, sh[j], sh[2 + j]);
        mma_bf16_16816(ca[j], kl, sh[j], sh[2 + j]);
        mma_bf16_16816(cp[j], ql, sh[j], sh[2 + j]);
        mma_bf16_16816(ca[j], kh, sl[j], sl[2 + j]);
        mma_bf16_16816(cp[j], qh, sl[j], sl[2 + j]);
      }
    } else {
      // token pairs one by one: this lane's entries (ta + 8 u, 8 j + kc + e), channels walked through shuffles
#pragma unroll 1
      for (int c = 0; c < 16; ++c) {
        const int v = c >> 3, src = (c & 7) >> 1, odd = c & 1;             // channel c lives in lanes 4 t + src
        float kt[2], qt[2], lt[2];
        const auto pick = [&](const float2& x) { return odd ? x.y : x.x; };
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          kt[u] = v ? pick(k[u][1]) : pick(k[u][0]);
          qt[u] = v ? pick(q[u][1]) : pick(q[u][0]);
          lt[u] = v ? pick(L[u][1]) : pick(L[u][0]);
        }
        float rk[2], rq[2], rl[2];           // of this lane's rows
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          rk[u] = __shfl_sync(0xffffffffu, kt[u], (lane & ~3) + src);
          rq[u] = __shfl_sync(0xffffffffu, qt[u], (lane & ~3) + src);
          rl[u] = __shfl_sync(0xffffffffu, lt[u], (lane & ~3) + src);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float sk = __shfl_sync(0xffffffffu, kt[j], 4 * (kc + e) + src);
            const float sl = __shfl_sync(0xffffffffu, lt[j], 4 * (kc + e) + src);
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              const float x = sk * exp2_flush(fminf(rl[u] - sl, 0.f));          // pairs with s > t are dropped later
              ca[j][2 * u + e] += rk[u] * x;
              cp[j][2 * u + e] += rq[u] * x;
            }
          }
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      part[warp][0][ta + (e >> 1) * 8][8 * j + kc + (e & 1)] = ca[j][e];
      part[warp][1][ta + (e >> 1) * 8][8 * j + kc + (e & 1)] = cp[j][e];
    }
  __syncthreads();
  {
    const int t = tid >> 4, s = tid & 15;
    float a = 0.f, q = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      a += part[w][0][t][s];
      q += part[w][1][t][s];
    }
    am[t][s] = s < t ? a * betas[t] : 0.f;
    if (s > t) q = 0.f;
    const bf16 hi = __float2bfloat16(q);
    bf16* pm = reinterpret_cast<bf16*>(blob + B::p);
    pm[tid] = hi;
    pm[kDC * kDC + tid] = __float2bfloat16(q - __bfloat162float(hi));
  }
  __syncthreads();
  if (tid < kDC) {                           // column tid of the inverse by forward substitution
    float x[kDC];
    bf16* mm = reinterpret_cast<bf16*>(blob + B::m);
    const float bt = betas[tid];
#pragma unroll
    for (int t = 0; t < kDC; ++t) {
      float y = t == tid ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < t; ++s) y -= am[t][s] * x[s];
      x[t] = y;
      const bf16 hi = __float2bfloat16(y * bt);
      mm[t * kDC + tid] = hi;
      mm[kDC * kDC + t * kDC + tid] = __float2bfloat16(y * bt - __bfloat162float(hi));
    }
  }
}

// grid (slices of 64 columns, heads, sequences)
template <int DK>
__global__ void __launch_bounds__(32 * kDWarps, DK > 128 ? 1 : 2) delta_chunk_kernel(DeltaChunk d) {
  using B = ChunkBlob<DK>;
  constexpr int CH = DK / 8, COLS = kDWarps * 16, VLD = COLS + 4, NT = 32 * kDWarps;
  constexpr int STAGE = (B::bytes + kDC * VLD * 4 + 127) / 128 * 128;
  const DeltaScan& p = d.s;
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c0 = blockIdx.x * COLS, dk = p.dk;
  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q[b], n_all = p.cu_q[b + 1] - row0, slot = p.slots[b];
  if (n_all <= 0 || slot < 0) return;
  const bool fresh = p.kv_lens[b] == n_all, works = c0 + warp * 16 < p.dv;
  float* S = p.state + (((int64_t)slot * p.H + h) * dk) * p.dvp;
  const int vloc = warp * 16 + (lane >> 2), vrow = c0 + vloc, kc = (lane & 3) * 2;
  float acc[DK / 8][4];                      // S^T: rows (value columns) lane / 4, + 8; key channels 8 nt + kc, + 1
#pragma unroll
  for (int nt = 0; nt < DK / 8; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = nt * 8 + kc + (e & 1), v = vrow + (e >> 1) * 8;
      acc[nt][e] = (!fresh && c < dk && v < p.dv) ? S[(int64_t)c * p.dvp + v] : 0.f;
    }
  const int chunks = (n_all + kDC - 1) / kDC;
  const uint8_t* blobs = d.blobs + (chunk_slot(row0, b, 0) * p.H + h) * B::bytes;
  const auto load = [&](int j) {
    if (j < chunks) {
      const uint32_t st = sb + (j % kDStages) * STAGE;
      const uint8_t* src = blobs + (int64_t)j * p.H * B::bytes;
      for (int i = tid; i < B::bytes / 16; i += NT) cp_async16(st + i * 16, src + i * 16, true);
      for (int i = tid; i < kDC * (COLS / 4); i += NT) {
        const int r = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
        const bool ok = j * kDC + r < n_all && c0 + c < p.dvp;
        cp_async16(st + B::bytes + (r * VLD + c) * 4,
                   p.vn + (ok ? ((int64_t)(row0 + j * kDC + r) * p.H + h) * p.dvp + c0 + c : 0), ok);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < kDStages - 1; ++s) load(s);
  const int arow = (lane & 7) + (((lane >> 3) & 1) << 3), acb = lane >> 4;
  const int brow = (lane & 7) + ((lane >> 4) << 3), bcb = (lane >> 3) & 1;
  for (int j = 0; j < chunks; ++j) {
    const int n = min(kDC, n_all - j * kDC);
    cp_async_wait<kDStages - 2>();
    __syncthreads();                         // chunk j is here, and everybody is done with the stage that is filled next
    load(j + kDStages - 1);
    if (!works) continue;
    const uint32_t st = sb + (j % kDStages) * STAGE;
    const uint8_t* stp = smem + (j % kDStages) * STAGE;
    float w[2][4], wl[2][4], o[2][4], ol[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) w[i][e] = wl[i][e] = o[i][e] = ol[i][e] = 0.f;
    // ---- W^T = S^T (k 2^L)^T, O^T = S^T (q 2^L)^T
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t kh[4], kl[4], qh[4], ql[4], hi[4], lo[4];
      const uint32_t at = st + swz<CH>(brow, kk * 2 + bcb);
      ldmatrix_x4(kh[0], kh[1], kh[2], kh[3], at + B::kt);
      ldmatrix_x4(kl[0], kl[1], kl[2], kl[3], at + B::kt + B::tile);
      ldmatrix_x4(qh[0], qh[1], qh[2], qh[3], at + B::qt);
      ldmatrix_x4(ql[0], ql[1], ql[2], ql[3], at + B::qt + B::tile);
      split_pack(acc[2 * kk][0], acc[2 * kk][1], hi[0], lo[0]);
      split_pack(acc[2 * kk][2], acc[2 * kk][3], hi[1], lo[1]);
      split_pack(acc[2 * kk + 1][0], acc[2 * kk + 1][1], hi[2], lo[2]);
      split_pack(acc[2 * kk + 1][2], acc[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mma_bf16_16816(w[i], hi, kh[2 * i], kh[2 * i + 1]);
        mma_bf16_16816(o[i], hi, qh[2 * i], qh[2 * i + 1]);
        mma_bf16_16816(wl[i], lo, kh[2 * i], kh[2 * i + 1]);
        mma_bf16_16816(ol[i], lo, qh[2 * i], qh[2 * i + 1]);
        mma_bf16_16816(wl[i], hi, kl[2 * i], kl[2 * i + 1]);
        mma_bf16_16816(ol[i], hi, ql[2 * i], ql[2 * i + 1]);
      }
    }
    // ---- U^T = (V - W)^T M^T
    const float* vs = reinterpret_cast<const float*>(stp + B::bytes);
    uint32_t rh[4], rl[4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float* v = vs + (8 * i + kc) * VLD + vloc + 8 * u;
        split_pack(v[0] - (w[i][2 * u] + wl[i][2 * u]), v[VLD] - (w[i][2 * u + 1] + wl[i][2 * u + 1]), rh[2 * i + u], rl[2 * i + u]);
      }
    float uu[2][4];
    uint32_t mh[4], ml[4], uh[4], ul[4];
    const uint32_t small = (uint32_t)(brow * kDC * 2 + bcb * 16);
    ldmatrix_x4(mh[0], mh[1], mh[2], mh[3], st + B::m + small);
    ldmatrix_x4(ml[0], ml[1], ml[2], ml[3], st + B::m + kDC * kDC * 2 + small);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
      for (int e = 0; e < 4; ++e) uu[i][e] = 0.f;
      mma_bf16_16816(uu[i], rh, mh[2 * i], mh[2 * i + 1]);
      mma_bf16_16816(uu[i], rl, mh[2 * i], mh[2 * i + 1]);
      mma_bf16_16816(uu[i], rh, ml[2 * i], ml[2 * i + 1]);
      split_pack(uu[i][0], uu[i][1], uh[2 * i], ul[2 * i]);
      split_pack(uu[i][2], uu[i][3], uh[2 * i + 1], ul[2 * i + 1]);
    }
    // ---- O^T += U^T P^T
    ldmatrix_x4(mh[0], mh[1], mh[2], mh[3], st + B::p + small);
    ldmatrix_x4(ml[0], ml[1], ml[2], ml[3], st + B::p + kDC * kDC * 2 + small);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mma_bf16_16816(o[i], uh, mh[2 * i], mh[2 * i + 1]);
      mma_bf16_16816(ol[i], ul, mh[2 * i], mh[2 * i + 1]);
      mma_bf16_16816(ol[i], uh, ml[2 * i], ml[2 * i + 1]);
    }
    // ---- S^T <- 2^(L_end) S^T + U^T (k 2^(L_end - L))
    const float* ge = reinterpret_cast<const float*>(stp + B::end);
#pragma unroll
    for (int nt = 0; nt < DK / 8; ++nt) {
      const float2 f = *reinterpret_cast<const float2*>(ge + nt * 8 + kc);
      acc[nt][0] *= f.x; acc[nt][1] *= f.y; acc[nt][2] *= f.x; acc[nt][3] *= f.y;
    }
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t kh[4], kl[4];
      const uint32_t at = st + B::kc + swz<CH>(arow, kk * 2 + acb);
      ldmatrix_x4_trans(kh[0], kh[1], kh[2], kh[3], at);
      ldmatrix_x4_trans(kl[0], kl[1], kl[2], kl[3], at + B::tile);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mma_bf16_16816(acc[2 * kk + i], uh, kh[2 * i], kh[2 * i + 1]);
        mma_bf16_16816(acc[2 * kk + i], ul, kh[2 * i], kh[2 * i + 1]);
        mma_bf16_16816(acc[2 * kk + i], uh, kl[2 * i], kl[2 * i + 1]);
      }
    }
    const int64_t row = row0 + j * kDC;
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = 8 * i + kc + (e & 1), v = vrow + (e >> 1) * 8;
        if (t < n && v < p.dv) p.o[((row + t) * p.H + h) * p.dv + v] = o[i][e] + ol[i][e];
      }
  }
  cp_async_wait<0>();
  if (!works) return;
#pragma unroll
  for (int nt = 0; nt < DK / 8; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = nt * 8 + kc + (e & 1), v = vrow + (e >> 1) * 8;
      if (c < dk && v < p.dvp) S[(int64_t)c * p.dvp + v] = acc[nt][e];
    }
}

template <int DK>
static int launch_delta_chunk(const DeltaChunk& d, int n_seqs, int max_q_len, cudaStream_t s) {
  using B = ChunkBlob<DK>;
  constexpr int COLS = kDWarps * 16;
  launch_pdl(delta_chunk_prep_kernel<DK>, dim3((max_q_len + kDC - 1) / kDC, d.s.H, n_seqs), dim3(256), 0, s, d);
  const int rc = XLLM_LAUNCH_CHECK();
  if (rc != 0) return rc;
  const size_t smem = (size_t)kDStages * ((B::bytes + kDC * (COLS + 4) * 4 + 127) / 128 * 128);
  const cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  launch_pdl(delta_chunk_kernel<DK>, dim3((d.s.dv + COLS - 1) / COLS, d.s.H, n_seqs), dim3(32 * kDWarps), smem, s, d);
  return XLLM_LAUNCH_CHECK();
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

XLLM_API int64_t xllm_delta_chunk_bytes(int rows, int n_seqs, int H, int dk) {
  using namespace xllm;
  const int64_t one = dk <= 64 ? ChunkBlob<64>::bytes : (dk <= 128 ? ChunkBlob<128>::bytes : ChunkBlob<256>::bytes);
  return ((int64_t)rows / kDC + n_seqs + 1) * H * one;
}

// dtype: 0 bf16, 1 fp32 (projection rows, weights, ring, finished rows).
//   state [slots, H, dk, dvp] fp32, dvp = dv rounded up to 4;  ring [slots, taps, 2 G dk + H dv]
//   q, k, v, r: column blocks of rows with stride ld;  zb fp32 [rows, zb_ld]
// qn, kn [rows, G, dkp], vn [rows, H, dvp], gn [rows, H, dkp] are fp32 scratch (dkp = dk rounded up to 4; gn comes with
// zeros behind dk).
// mode 0: one token per sequence (sequence s is row s, cu_q counts up by one): gate, norm_w, out are used; dk <= 256, dv <= 128
// mode 1: rows [row0, rows) by cu_q, the raw fp32 outputs go to o [rows, H, dv];  dk <= 512
// mode 2: the same in chunks of 16 tokens, no sequence longer than max_q_len rows; dk <= 256;
//         blobs: scratch of xllm_delta_chunk_bytes(rows, n_seqs, H, dk) bytes
XLLM_API int xllm_delta_rule(void* state, void* ring, const void* slots, const void* cu_q, const void* kv_lens, const void* q,
                             const void* k, const void* v, const void* r, int64_t ld, const void* zb, int64_t zb_ld,
                             const void* conv_w, const void* a2, const void* dt_bias, const void* a_log, const void* gate,
                             int64_t gate_ld, const void* norm_w, void* out, int64_t out_ld, void* qn, void* kn, void* vn,
                             void* gn, void* o, int n_seqs, int rows, int row0, int H, int G, int dk, int dv, int taps,
                             int rank, float q_scale, float eps, int dtype, int mode, void* blobs, int max_q_len, void* stream) {
  using namespace xllm;
  if (n_seqs == 0 || rows - row0 <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || dk <= 0 || dk > 512 || dv <= 0 || taps <= 0 || rank <= 0)
    return (int)cudaErrorInvalidValue;
  if (mode == 0 && (dk > 256 || dv > 128)) return (int)cudaErrorInvalidValue;
  if (mode == 2 && (dk > 256 || blobs == nullptr || max_q_len <= 0)) return (int)cudaErrorInvalidValue;
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
    p.log_decay = mode == 2;
    p.write_ring = mode == 0 && taps > 1;
    if ((rc = launch_channel_decay(p, s)) != 0) return;
    const auto al = [](const void* x, size_t a) { return (((uintptr_t)x) & (a - 1)) == 0; };
    const size_t va = 4 * sizeof(T);
    const bool v4 = dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && al(q, va) && al(k, va) && al(v, va) && al(ring, va) &&
                    al(conv_w, va);
    const int run = v4 && taps <= 4 && dk <= 128 && dv <= 128 ? (mode == 0 ? 1 : 4) : 0;
    const int64_t warps = (int64_t)(run > 0 ? (rows - row0 + run - 1) / run : rows - row0) * (2 * G + H);
    const dim3 grid((unsigned)((warps + 7) / 8));
    if (run == 1) launch_pdl(conv_heads_run_kernel<T, 1>, grid, dim3(256), 0, s, p);
    else if (run > 1) launch_pdl(conv_heads_run_kernel<T, 4>, grid, dim3(256), 0, s, p);
    else if (v4) launch_pdl(conv_heads_kernel<T, 4>, grid, dim3(256), 0, s, p);
    else launch_pdl(conv_heads_kernel<T, 1>, grid, dim3(256), 0, s, p);
    if ((rc = XLLM_LAUNCH_CHECK()) != 0) return;
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
    if (taps > 1) {
      launch_pdl(conv_ring_kernel<T>, dim3((unsigned)((p.channels() + 255) / 256), n_seqs), dim3(256), 0, s, p);
      if ((rc = XLLM_LAUNCH_CHECK()) != 0) return;
    }
    DeltaScan d{p.state, p.slots, p.cu_q, p.kv_lens, p.qn, p.kn, p.vn, p.gn, p.zb, zb_ld, p.o, H, G, dk, dv, p.dkp, p.dvp};
    if (mode == 2) {
      const DeltaChunk c{d, (uint8_t*)blobs};
      if (dk <= 64) rc = launch_delta_chunk<64>(c, n_seqs, max_q_len, s);
      else if (dk <= 128) rc = launch_delta_chunk<128>(c, n_seqs, max_q_len, s);
      else rc = launch_delta_chunk<256>(c, n_seqs, max_q_len, s);
      return;
    }
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
