// What lies between a fused projection and paged attention, in one pass over q, k and v, any head size up to 512, bf16 or
// fp32, every step optional:
//   a short causal convolution over time per channel of q, k and v,
//   a per-head RMS norm of q and k with a weight shared by the heads,
//   rotary positions on the first `rot` elements of q and k,
//   a per-head RMS norm of q and k without a weight;
// or, behind the convolution and without rotation (xllm_conv_row_norm_kv):
//   an RMS norm of all of q, and one of all of k, with a weight per element,
//   a per-head RMS norm of the values without a weight.
// k goes to the paged K cache and the values (any column block of the row: their own projection, or the keys as projected)
// to the V cache.
//
// The sibling of rope_kv.cu (weighted norm and rotation, power-of-two head sizes).  Heads may be stored wider than they are
// (d_pad >= d, zero filled): the attention kernels take head sizes 64, 128 and 256.  The generic kernel has one warp per
// (token, head), a lane owns element pairs.  The convolution keeps a sequence's last inputs in a ring (short_conv.cuh); a
// sequence with one row in the batch stores it here, longer portions in a launch behind this one.
#include "short_conv.cuh"

namespace xllm {

template <typename T>
struct RopeNormParams {
  const T *q, *k, *v;       // column blocks of the projection rows (row stride ld)
  int64_t ld;
  T* q_out;                 // [T, nq, d_pad]
  T* k_cache;               // [n_blocks, nkv, page, d_pad]
  T* v_cache;
  const float* cos_sin;     // [max_pos, rot]: cos | sin, or null
  const int64_t* positions;
  const int32_t* slots;     // < 0: nothing is cached
  int tokens, nq, nkv, d, dv, d_pad, rot, page, interleaved, unit_norm;
  int64_t max_pos;
  float eps;
  const T *q_w, *k_w;        // [d] weights of the norm ahead of the rotation, or null
  // short convolution (taps 0: none); channels are q | k | v
  const T* conv_w;           // [taps, channels], the last row belongs to the current token
  T* ring;                   // [state slots, taps, channels]
  const int32_t *state_slots, *cu_q, *kv_lens;      // [n_seqs], [n_seqs + 1], [n_seqs]
  int n_seqs, taps;
  __host__ __device__ int64_t channels() const { return (int64_t)(nq + nkv) * d + (int64_t)nkv * dv; }
};

// where a token row stands in its sequence
struct ConvPlace {
  int slot, back, pos, alone;          // state slot (-1: no sequence), rows of the sequence ahead of it in the batch, position
};
template <typename T>
__device__ __forceinline__ ConvPlace conv_place(const RopeNormParams<T>& p, int row) {
  ConvPlace c{-1, 0, 0, 0};
  const int b = seq_of_row(p.cu_q, p.n_seqs, row);
  if (b < 0 || p.kv_lens[b] <= 0) return c;
  c.slot = p.state_slots[b];
  c.back = row - p.cu_q[b];
  c.pos = p.kv_lens[b] - (p.cu_q[b + 1] - row);
  c.alone = p.cu_q[b + 1] - p.cu_q[b] == 1;
  return c;
}
// one channel of one row behind the convolution; x: its place in the row, ch: its number among the channels
template <typename T>
__device__ __forceinline__ float conv_one(const RopeNormParams<T>& p, const ConvPlace& c, const T* x, int64_t ch) {
  if (c.slot < 0) return 0.f;
  const int64_t C = p.channels();
  T* ring = p.ring + (int64_t)c.slot * p.taps * C + ch;
  float y = 0.f;
  for (int b = 0; b < p.taps && b <= c.pos; ++b)
    y += to_f32(b <= c.back ? x[-b * p.ld] : ring[(c.pos - b) % p.taps * C]) * to_f32(p.conv_w[(p.taps - 1 - b) * C + ch]);
  if (c.alone) ring[c.pos % p.taps * C] = x[0];
  return y;
}

constexpr int kPairs = 8;   // pairs per lane: d <= 512

template <typename T>
__global__ void __launch_bounds__(256) rope_norm_kv_kernel(RopeNormParams<T> p) {
  const int lane = threadIdx.x & 31;
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int heads = p.nq + p.nkv;
  pdl_wait();
  pdl_launch_dependents();
  if (item >= (int64_t)p.tokens * heads) return;
  const int64_t t = item / heads;
  const int h = (int)(item - t * heads);
  const bool is_q = h < p.nq;
  const int g = is_q ? h : h - p.nq;
  const T* src = (is_q ? p.q : p.k) + t * p.ld + (int64_t)g * p.d;
  const bool conv = p.taps > 0;
  const int64_t ch = (int64_t)h * p.d;
  ConvPlace place{};
  if (conv) place = conv_place(p, (int)t);
  const auto in = [&](int i) { return conv ? conv_one(p, place, src + i, ch + i) : to_f32(src[i]); };
  const T* w = is_q ? p.q_w : p.k_w;
  const int half = p.rot >> 1;
  const float* cs = nullptr;
  if (p.cos_sin != nullptr) {
    int64_t pos = p.positions[t];
    pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
    cs = p.cos_sin + pos * p.rot;
  }
  // pair n of the head: the rotated pairs first, then neighbours of the part that passes unchanged
  const int n_pairs = (p.d + 1) >> 1;
  float a[kPairs], b[kPairs];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kPairs; ++i) {
    a[i] = b[i] = 0.f;
    const int n = lane + 32 * i;
    if (n >= n_pairs) continue;
    int i0, i1;
    if (n < half && !p.interleaved) { i0 = n; i1 = n + half; }
    else { i0 = 2 * n; i1 = 2 * n + 1; }
    a[i] = in(i0);
    b[i] = i1 < p.d ? in(i1) : 0.f;
    ss += a[i] * a[i] + b[i] * b[i];
  }
  if (w != nullptr) {
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.d + p.eps);
#pragma unroll
    for (int i = 0; i < kPairs; ++i) {
      const int n = lane + 32 * i;
      if (n >= n_pairs) continue;
      const bool split = n < half && !p.interleaved;
      const int i0 = split ? n : 2 * n, i1 = split ? n + half : 2 * n + 1;
      a[i] *= inv * to_f32(w[i0]);
      if (i1 < p.d) b[i] *= inv * to_f32(w[i1]);
    }
  }
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kPairs; ++i) {
    const int n = lane + 32 * i;
    if (n < half && cs != nullptr) {
      const float c = cs[n], s = cs[half + n];
      const float u = a[i], v = b[i];
      a[i] = u * c - v * s;
      b[i] = v * c + u * s;
    }
    ss += a[i] * a[i] + b[i] * b[i];
  }
  float inv = 1.f;
  if (p.unit_norm) inv = 1.f / sqrtf(warp_sum(ss) / (float)p.d + p.eps);
  const int slot = is_q ? 0 : p.slots[t];
  if (!is_q && slot < 0 && !conv) return;
  const bool cached = is_q || slot >= 0;
  const int64_t blk = slot < 0 ? 0 : slot / p.page;
  const int off = slot - (int)blk * p.page;
  const int64_t crow = ((blk * p.nkv + g) * p.page + off) * (int64_t)p.d_pad;
  T* dst = is_q ? p.q_out + (t * p.nq + g) * p.d_pad : p.k_cache + crow;
#pragma unroll
  for (int i = 0; i < kPairs; ++i) {
    const int n = lane + 32 * i;
    if (n >= n_pairs || !cached) continue;
    int i0, i1;
    if (n < half && !p.interleaved) { i0 = n; i1 = n + half; }
    else { i0 = 2 * n; i1 = 2 * n + 1; }
    dst[i0] = from_f32<T>(a[i] * inv);
    if (i1 < p.d) dst[i1] = from_f32<T>(b[i] * inv);
  }
  for (int i = p.d + lane; i < p.d_pad && cached; i += 32) dst[i] = from_f32<T>(0.f);
  if (!is_q) {
    const T* vs = p.v + t * p.ld + (int64_t)g * p.dv;
    const int64_t vch = (int64_t)(p.nq + p.nkv) * p.d + (int64_t)g * p.dv;
    T* vd = p.v_cache + crow;
    for (int i = lane; i < p.d_pad; i += 32) {
      T v = from_f32<T>(0.f);
      if (i < p.dv) v = conv ? from_f32<T>(conv_one(p, place, vs + i, vch + i)) : vs[i];
      if (cached) vd[i] = v;
    }
  }
}

// bf16 heads of 8, 16, ... 256 elements with aligned rows: one CTA per token, a thread owns eight contiguous elements
// of up to four heads, whose 16-byte loads are all issued first (the layout of rope_kv.cu).
constexpr int kVecHeads = 4;

// NORM: the weighted norm; SAME: value heads of d elements.
template <bool NORM, bool SAME>
__global__ void __launch_bounds__(256) rope_norm_kv_vec_kernel(RopeNormParams<bf16> p) {
  const int tph = p.d >> 3, per_pass = 256 / tph;
  const int local = threadIdx.x / tph, g = threadIdx.x - local * tph, e0 = g * 8;
  const int heads = p.nq + p.nkv, half = p.rot >> 1;
  const int64_t t = blockIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  const bool turns = p.cos_sin != nullptr && e0 < p.rot;
  float c[8], sn[8];
  if (turns) {
    int64_t pos = p.positions[t];
    pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
    const float* cs = p.cos_sin + pos * p.rot;
    if (p.interleaved) {
      load_f32<4>(cs + (e0 >> 1), c);
      load_f32<4>(cs + half + (e0 >> 1), sn);
    } else {
      const int ci = e0 < half ? e0 : e0 - half;
      load_f32<8>(cs + ci, c);
      load_f32<8>(cs + half + ci, sn);
    }
  }
  const int slot = p.slots[t];
  const int64_t blk = slot / p.page;
  const int off = slot - (int)blk * p.page;
  for (int h0 = 0; h0 < heads; h0 += per_pass * kVecHeads) {
    bf16x8 raw[kVecHeads], val[kVecHeads];
#pragma unroll
    for (int u = 0; u < kVecHeads; ++u) {
      const int h = h0 + u * per_pass + local;
      if (h >= heads) continue;
      const bool is_q = h < p.nq;
      raw[u] = *reinterpret_cast<const bf16x8*>((is_q ? p.q : p.k) + t * p.ld + (int64_t)(is_q ? h : h - p.nq) * p.d + e0);
      if (SAME && !is_q && p.v != p.k)
        val[u] = *reinterpret_cast<const bf16x8*>(p.v + t * p.ld + (int64_t)(h - p.nq) * p.d + e0);
    }
#pragma unroll
    for (int u = 0; u < kVecHeads; ++u) {
      const int h = h0 + u * per_pass + local;
      const bool active = h < heads;               // whole heads are active or not together
      float x[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = 0.f;
      if (active) unpack8(raw[u], x);
      if constexpr (NORM) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
        for (int o = tph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.f / sqrtf(ss / (float)p.d + p.eps);
        float w[8];
        load_f32<8>((h < p.nq ? p.q_w : p.k_w) + e0, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] *= inv * w[j];
      }
      if (p.cos_sin != nullptr) {
        if (p.interleaved) {
          if (turns) {
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
              const float a = x[j], b = x[j + 1];
              x[j] = a * c[j >> 1] - b * sn[j >> 1];
              x[j + 1] = b * c[j >> 1] + a * sn[j >> 1];
            }
          }
        } else {
          float other[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) other[j] = __shfl_xor_sync(0xffffffffu, x[j], half >> 3);
          if (turns) {
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = e0 < half ? x[j] * c[j] - other[j] * sn[j] : x[j] * c[j] + other[j] * sn[j];
          }
        }
      }
      if (p.unit_norm) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
        for (int o = tph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.f / sqrtf(ss / (float)p.d + p.eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] *= inv;
      }
      if (!active) continue;
      const bool is_q = h < p.nq;
      if (!is_q && slot < 0) continue;
      const int kvh = h - p.nq;
      const int64_t crow = ((blk * p.nkv + kvh) * p.page + off) * (int64_t)p.d_pad;
      bf16* dst = is_q ? p.q_out + (t * p.nq + h) * p.d_pad : p.k_cache + crow;
      *reinterpret_cast<bf16x8*>(dst + e0) = pack8(x);
      if (SAME && !is_q) *reinterpret_cast<bf16x8*>(p.v_cache + crow + e0) = p.v != p.k ? val[u] : raw[u];
      for (int z = p.d + e0; z < p.d_pad; z += p.d) {
        *reinterpret_cast<uint4*>(dst + z) = make_uint4(0, 0, 0, 0);
        if (SAME && !is_q) *reinterpret_cast<uint4*>(p.v_cache + crow + z) = make_uint4(0, 0, 0, 0);
      }
    }
  }
  if (SAME || slot < 0) return;
  const int vph = p.d_pad >> 3;                        // vectors of a stored value head
  for (int n = threadIdx.x; n < p.nkv * vph; n += 256) {
    const int h = n / vph, e = (n - h * vph) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (e < p.dv) v = *reinterpret_cast<const uint4*>(p.v + t * p.ld + (int64_t)h * p.dv + e);
    *reinterpret_cast<uint4*>(p.v_cache + ((blk * p.nkv + h) * p.page + off) * (int64_t)p.d_pad + e) = v;
  }
}

// The same sizes behind a convolution of up to four taps (rotate-half layout, no weightless norm): a CTA takes RUN token
// rows and 256 vectors of V channels; a thread reads every input of its vector once, some rows ahead, and keeps the last
// ones in registers.  grid (runs, parts): the first `qk_parts` parts are q and k, the others v.
constexpr int kMaxTaps = 4;
constexpr int kConvRun = 4;

template <int RUN, int V>
__global__ void __launch_bounds__(256, V == 4 ? 4 : 1) conv_rope_kv_kernel(RopeNormParams<bf16> p, int qk_parts) {
  constexpr int AHEAD = RUN < 4 ? RUN : 4;
  struct __align__(V * 2) Vec { bf16 v[V]; };
  __shared__ ConvPlace place[RUN];
  __shared__ int64_t cache_row[RUN];                                 // of kv head 0; negative: nothing is cached
  __shared__ int64_t angle_row[RUN];
  const int first = blockIdx.x * RUN;
  pdl_wait();
  pdl_launch_dependents();
  const bool is_v = (int)blockIdx.y >= qk_parts;
  const int size = is_v ? p.dv : p.d, per = size / V;                // vectors of a head
  const int n = ((int)blockIdx.y - (is_v ? qk_parts : 0)) * 256 + threadIdx.x;
  const int heads = is_v ? p.nkv : p.nq + p.nkv;
  const bool on = n < heads * per;                                   // whole heads are on or not together
  const int h = on ? n / per : 0, e0 = on ? (n - h * per) * V : 0;
  const bool is_q = !is_v && h < p.nq;
  const int kvh = is_v ? h : h - p.nq;
  const int64_t C = p.channels(), ch = (is_v ? (int64_t)(p.nq + p.nkv) * p.d : 0) + (int64_t)h * size + e0;
  const bf16* x = (is_v ? p.v + (int64_t)h * size : (is_q ? p.q + (int64_t)h * size : p.k + (int64_t)kvh * size)) + e0;
  const auto fetch = [&](int row) {
    Vec f{};
    if (on && row >= 0 && row < p.tokens) f = *reinterpret_cast<const Vec*>(x + row * p.ld);
    return f;
  };
  Vec raw[AHEAD], old[kMaxTaps - 1];
#pragma unroll
  for (int r = 0; r < AHEAD; ++r) raw[r] = fetch(first + r);
#pragma unroll
  for (int b = 1; b < kMaxTaps; ++b) old[b - 1] = RUN > 1 && b < p.taps ? fetch(first - b) : Vec{};
  if (threadIdx.x < RUN) {
    const int row = first + threadIdx.x;
    ConvPlace c{-1, 0, 0, 0};
    int64_t pos = 0, at = -1;
    if (row < p.tokens) {
      c = conv_place(p, row);
      const int cs = p.slots[row];
      if (cs >= 0) at = (int64_t)(cs / p.page) * p.nkv * p.page + cs % p.page;
      if (p.cos_sin != nullptr) pos = p.positions[row];
    }
    place[threadIdx.x] = c;
    cache_row[threadIdx.x] = at;
    angle_row[threadIdx.x] = (pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos)) * p.rot;
  }
  float w[kMaxTaps][V], win[kMaxTaps][V];                            // win[b]: the input b tokens back
#pragma unroll
  for (int b = 0; b < kMaxTaps; ++b) {
#pragma unroll
    for (int j = 0; j < V; ++j) {
      w[b][j] = 0.f;
      win[b][j] = b > 0 ? __bfloat162float(old[b - 1].v[j]) : 0.f;
    }
    if (on && b < p.taps) load_f32<V>(p.conv_w + (p.taps - 1 - b) * C + ch, w[b]);
  }
  const int half = p.rot >> 1;
  const bool turns = !is_v && p.cos_sin != nullptr && e0 < p.rot;
  const int angle = e0 < half ? e0 : e0 - half;
  const float sign = e0 < half ? -1.f : 1.f;
  __syncthreads();
#pragma unroll
  for (int r = 0; r < RUN; ++r) {
    const int row = first + r;
    if (row >= p.tokens) break;
#pragma unroll
    for (int j = 0; j < V; ++j) win[0][j] = __bfloat162float(raw[r % AHEAD].v[j]);
    if (r + AHEAD < RUN) raw[r % AHEAD] = fetch(row + AHEAD);
    const ConvPlace c = place[r];
    const int64_t at = cache_row[r];
    float y[V];
    if (c.slot >= 0) {
      if (c.back < kMaxTaps - 1) {                                   // inputs of earlier steps, or of none
        const bf16* ring = p.ring + (int64_t)c.slot * p.taps * C + ch;
#pragma unroll
        for (int b = 1; b < kMaxTaps; ++b) {
          if (b <= c.back) continue;
          if (on && b < p.taps && b <= c.pos) load_f32<V>(ring + (c.pos - b) % p.taps * C, win[b]);
          else {
#pragma unroll
            for (int j = 0; j < V; ++j) win[b][j] = 0.f;
          }
        }
        if (c.alone && on) store_f32<V>(p.ring + ((int64_t)c.slot * p.taps + c.pos % p.taps) * C + ch, win[0]);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) {
        y[j] = win[0][j] * w[0][j];
#pragma unroll
        for (int b = 1; b < kMaxTaps; ++b) y[j] = fmaf(win[b][j], w[b][j], y[j]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) y[j] = 0.f;
    }
#pragma unroll
    for (int b = kMaxTaps - 1; b > 0; --b)
#pragma unroll
      for (int j = 0; j < V; ++j) win[b][j] = win[b - 1][j];
    if (!is_v) {
      if (p.q_w != nullptr) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < V; ++j) ss += y[j] * y[j];
        for (int o = per >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.f / sqrtf(ss / (float)p.d + p.eps);
        float f[V];
        load_f32<V>((is_q ? p.q_w : p.k_w) + e0, f);
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] *= inv * f[j];
      }
      if (p.cos_sin != nullptr) {
        float other[V];
#pragma unroll
        for (int j = 0; j < V; ++j) other[j] = __shfl_xor_sync(0xffffffffu, y[j], half / V);
        if (turns) {
          float co[V], si[V];
          const float* a = p.cos_sin + angle_row[r] + angle;
          load_f32<V>(a, co);
          load_f32<V>(a + half, si);
#pragma unroll
          for (int j = 0; j < V; ++j) y[j] = fmaf(y[j], co[j], sign * si[j] * other[j]);
        }
      }
    }
    if (!on || (!is_q && at < 0)) continue;
    const int64_t crow = (at + kvh * p.page) * p.d_pad;
    bf16* dst = is_v ? p.v_cache + crow : (is_q ? p.q_out + ((int64_t)row * p.nq + h) * p.d_pad : p.k_cache + crow);
    store_f32<V>(dst + e0, y);
    for (int z = size + e0; z < p.d_pad; z += size) *reinterpret_cast<Vec*>(dst + z) = Vec{};
  }
}

// the last inputs of every sequence with more than one row in the batch
template <typename T>
__global__ void __launch_bounds__(256) conv_keep_kernel(RopeNormParams<T> p) {
  const int b = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, slot = p.state_slots[b];
  const int64_t c = (int64_t)blockIdx.x * 256 + threadIdx.x, C = p.channels();
  if (n <= 1 || slot < 0 || c >= C) return;
  const int64_t q_end = (int64_t)p.nq * p.d, k_end = q_end + (int64_t)p.nkv * p.d;
  const T* x = c < q_end ? p.q + c : (c < k_end ? p.k + c - q_end : p.v + c - k_end);
  for (int i = max(0, n - (p.taps - 1)); i < n; ++i)
    p.ring[((int64_t)slot * p.taps + (p.kv_lens[b] - n + i) % p.taps) * C + c] = x[(int64_t)(first + i) * p.ld];
}

// Norms over whole rows.  One CTA takes RUN token rows one after another; a thread owns NV vectors of eight channels of q | k | v,
// keeps their last inputs in registers, and the sums of squares meet once per row: those of q and k through the
// warps, those of the values as one number per vector, so that every head adds its own in a fixed order.  portions: a sequence may
// have several rows.
constexpr int kRowThreads = 512;

template <int RUN, int NV>
__global__ void __launch_bounds__(kRowThreads) conv_row_norm_kernel(RopeNormParams<bf16> p, int portions) {
  __shared__ ConvPlace place[RUN];
  __shared__ int64_t cache_row[RUN];
  __shared__ float sums[2][2][kRowThreads / 32];
  extern __shared__ float vsum[];                                    // [2][value vectors]
  const int first = blockIdx.x * RUN, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nq = p.nq * p.d / 8, nk = p.nkv * p.d / 8, nv = p.nkv * p.dv / 8, n = nq + nk + nv;
  const int64_t C = (int64_t)n * 8;
  pdl_wait();
  pdl_launch_dependents();
  const bf16* src[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * kRowThreads;
    src[i] = v < nq ? p.q + v * 8 : (v < nq + nk ? p.k + (v - nq) * 8 : p.v + (v - nq - nk) * 8);
  }
  const auto fetch = [&](int i, int row) {
    bf16x8 f{};
    if ((int)threadIdx.x + i * kRowThreads < n && row >= 0 && row < p.tokens) f = *reinterpret_cast<const bf16x8*>(src[i] + row * p.ld);
    return f;
  };
  constexpr bool HOLD = NV == 1;                                     // weights stay in registers, else in L1
  const auto weight = [&](int i, int b) {
    const int v = threadIdx.x + i * kRowThreads;
    return v < n && b < p.taps ? *reinterpret_cast<const bf16x8*>(p.conv_w + (p.taps - 1 - b) * C + v * 8) : bf16x8{};
  };
  bf16x8 w[HOLD ? 1 : NV][HOLD ? kMaxTaps : 1], win[NV][kMaxTaps];   // win[b]: the input b tokens back
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    win[i][0] = fetch(i, first);
#pragma unroll
    for (int b = 0; b < kMaxTaps; ++b) {
      if constexpr (HOLD) w[i][b] = weight(i, b);
      if (b > 0) win[i][b] = portions && b < p.taps ? fetch(i, first - b) : bf16x8{};
    }
  }
  if (threadIdx.x < RUN) {
    const int row = first + threadIdx.x;
    ConvPlace c{-1, 0, 0, 0};
    int64_t at = -1;
    if (row < p.tokens) {
      c = conv_place(p, row);
      const int cs = p.slots[row];
      if (cs >= 0) at = (int64_t)(cs / p.page) * p.nkv * p.page + cs % p.page;
    }
    place[threadIdx.x] = c;
    cache_row[threadIdx.x] = at;
  }
  __syncthreads();
#pragma unroll 1
  for (int r = 0; r < RUN; ++r) {
    const int row = first + r;
    if (row >= p.tokens) break;
    const ConvPlace c = place[r];
    float y[NV][8], qs = 0.f, ks = 0.f;
    bf16x8 next[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = threadIdx.x + i * kRowThreads;
      next[i] = r + 1 < RUN ? fetch(i, row + 1) : bf16x8{};
#pragma unroll
      for (int j = 0; j < 8; ++j) y[i][j] = 0.f;
      if (c.slot >= 0 && v < n) {
        bf16* ring = p.ring + (int64_t)c.slot * p.taps * C + v * 8;
        if (c.back < kMaxTaps - 1) {                                 // inputs of earlier steps, or of none
#pragma unroll
          for (int b = 1; b < kMaxTaps; ++b) {
            if (b <= c.back) continue;
            win[i][b] = bf16x8{};
            if (b < p.taps && b <= c.pos) win[i][b] = *reinterpret_cast<const bf16x8*>(ring + (c.pos - b) % p.taps * C);
          }
          if (c.alone) *reinterpret_cast<bf16x8*>(ring + c.pos % p.taps * C) = win[i][0];
        }
        float ss = 0.f;
#pragma unroll
        for (int b = 0; b < kMaxTaps; ++b) {
          float f[8], g[8];
          unpack8(win[i][b], f);
          if constexpr (HOLD) unpack8(w[i][b], g);
          else unpack8(weight(i, b), g);
#pragma unroll
          for (int j = 0; j < 8; ++j) y[i][j] = fmaf(f[j], g[j], y[i][j]);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += y[i][j] * y[i][j];
        if (v < nq) qs += ss;
        else if (v < nq + nk) ks += ss;
        else vsum[(r & 1) * nv + v - nq - nk] = ss;
      } else if (v >= nq + nk && v < n) {
        vsum[(r & 1) * nv + v - nq - nk] = 0.f;
      }
#pragma unroll
      for (int b = kMaxTaps - 1; b > 0; --b) win[i][b] = win[i][b - 1];
      win[i][0] = next[i];
    }
    qs = warp_sum(qs);
    ks = warp_sum(ks);
    if (lane == 0) {
      sums[r & 1][0][warp] = qs;
      sums[r & 1][1][warp] = ks;
    }
    __syncthreads();
    qs = ks = 0.f;
#pragma unroll
    for (int i = 0; i < kRowThreads / 32; ++i) {
      qs += sums[r & 1][0][i];
      ks += sums[r & 1][1][i];
    }
    const float qi = 1.f / sqrtf(qs / (float)(p.nq * p.d) + p.eps), ki = 1.f / sqrtf(ks / (float)(p.nkv * p.d) + p.eps);
    const int64_t at = cache_row[r];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = threadIdx.x + i * kRowThreads;
      if (v >= n || (v >= nq && at < 0)) continue;
      const bool is_q = v < nq, is_v = v >= nq + nk;
      const int u = is_q ? v : (is_v ? v - nq - nk : v - nq), size = is_v ? p.dv : p.d;
      const int h = u * 8 / size, e = u * 8 - h * size;
      if (!is_v) {
        float g[8];
        load_f32<8>((is_q ? p.q_w : p.k_w) + u * 8, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[i][j] *= (is_q ? qi : ki) * g[j];
      } else {
        float ss = 0.f;
        for (int k = 0; k < p.dv / 8; ++k) ss += vsum[(r & 1) * nv + h * (p.dv / 8) + k];
        const float inv = 1.f / sqrtf(ss / (float)p.dv + p.eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[i][j] *= inv;
      }
      bf16* dst = is_q ? p.q_out + ((int64_t)row * p.nq + h) * p.d_pad : (is_v ? p.v_cache : p.k_cache) + (at + h * p.page) * p.d_pad;
      store_f32<8>(dst + e, y[i]);
      for (int z = size + e; z < p.d_pad; z += size) *reinterpret_cast<uint4*>(dst + z) = make_uint4(0, 0, 0, 0);
    }
  }
}

// any sizes and taps: one CTA per token row, the convolution is computed twice
template <typename T>
__global__ void __launch_bounds__(256) conv_row_norm_any_kernel(RopeNormParams<T> p) {
  __shared__ float red[32];
  const int row = blockIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  const ConvPlace c = conv_place(p, row);
  ConvPlace look = c;
  look.alone = 0;                                                    // the ring row is stored in the second pass
  const int64_t nq = (int64_t)p.nq * p.d, nk = (int64_t)p.nkv * p.d;
  const int slot = p.slots[row];
  const int64_t at = slot >= 0 ? (int64_t)(slot / p.page) * p.nkv * p.page + slot % p.page : 0;
  int64_t ch = 0;
  for (int part = 0; part < 2; ++part) {
    const int64_t size = part == 0 ? nq : nk;
    const T* x = (part == 0 ? p.q : p.k) + row * p.ld;
    const T* w = part == 0 ? p.q_w : p.k_w;
    float ss = 0.f;
    for (int64_t i = threadIdx.x; i < size; i += 256) {
      const float y = conv_one(p, look, x + i, ch + i);
      ss += y * y;
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)size + p.eps);
    for (int64_t i = threadIdx.x; i < size; i += 256) {
      const float y = conv_one(p, c, x + i, ch + i);
      const int h = (int)(i / p.d), e = (int)(i - (int64_t)h * p.d);
      if (part == 0) p.q_out[((int64_t)row * p.nq + h) * p.d_pad + e] = from_f32<T>(y * inv * to_f32(w[i]));
      else if (slot >= 0) p.k_cache[(at + h * p.page) * p.d_pad + e] = from_f32<T>(y * inv * to_f32(w[i]));
    }
    const int heads = part == 0 ? p.nq : p.nkv, gap = p.d_pad - p.d;
    for (int i = threadIdx.x; i < heads * gap; i += 256) {
      const int h = i / gap, e = p.d + i - h * gap;
      if (part == 0) p.q_out[((int64_t)row * p.nq + h) * p.d_pad + e] = from_f32<T>(0.f);
      else if (slot >= 0) p.k_cache[(at + h * p.page) * p.d_pad + e] = from_f32<T>(0.f);
    }
    ch += size;
  }
  const int lane = threadIdx.x & 31;
  for (int h = threadIdx.x >> 5; h < p.nkv; h += 8) {
    const T* x = p.v + row * p.ld + (int64_t)h * p.dv;
    const int64_t vch = ch + (int64_t)h * p.dv;
    float ss = 0.f;
    for (int i = lane; i < p.dv; i += 32) {
      const float y = conv_one(p, look, x + i, vch + i);
      ss += y * y;
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
    T* dst = p.v_cache + (at + h * p.page) * p.d_pad;
    for (int i = lane; i < p.d_pad; i += 32) {
      const float y = i < p.dv ? conv_one(p, c, x + i, vch + i) : 0.f;
      if (slot >= 0) dst[i] = from_f32<T>(y * inv);
    }
  }
}

}  // namespace xllm

// dtype: 0 bf16, 1 fp32.  rot <= d, rot even.  dv: size of a value head (d where v is the key block).
// q_w, k_w: both or neither.  taps > 0: the convolution; conv_w .. kv_lens as in RopeNormParams, over all rows of the batch;
// long_portions: some sequence may have more than one row.
XLLM_API int xllm_rope_norm_kv(const void* q, const void* k, const void* v, int64_t ld, void* q_out, void* k_cache,
                               void* v_cache, const void* cos_sin, int64_t max_pos, const void* positions, const void* slots,
                               int tokens, int nq, int nkv, int d, int dv, int d_pad, int rot, int page, int interleaved, int unit_norm,
                               float eps, const void* q_w, const void* k_w, const void* conv_w, void* ring, const void* state_slots,
                               const void* cu_q, const void* kv_lens, int n_seqs, int taps, int long_portions, int dtype,
                               void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (d <= 0 || d > 64 * kPairs || d_pad < d || dv <= 0 || d_pad < dv || rot < 0 || rot > d || rot % 2 != 0 || page <= 0 || nq <= 0 || nkv <= 0 || (q_w == nullptr) != (k_w == nullptr))
    return (int)cudaErrorInvalidValue;
  if (taps < 0 || (taps > 0 && (conv_w == nullptr || ring == nullptr || state_slots == nullptr || cu_q == nullptr ||
                                kv_lens == nullptr || n_seqs <= 0)))
    return (int)cudaErrorInvalidValue;
  const int64_t items = (int64_t)tokens * (nq + nkv);
  const dim3 grid((unsigned)((items + 7) / 8)), block(256);
  cudaStream_t s = (cudaStream_t)stream;
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    RopeNormParams<T> p;
    p.q = (const T*)q; p.k = (const T*)k; p.v = (const T*)v; p.ld = ld; p.q_out = (T*)q_out; p.k_cache = (T*)k_cache;
    p.v_cache = (T*)v_cache; p.cos_sin = rot > 0 ? (const float*)cos_sin : nullptr; p.positions = (const int64_t*)positions;
    p.slots = (const int32_t*)slots; p.tokens = tokens; p.nq = nq; p.nkv = nkv; p.d = d; p.dv = dv; p.d_pad = d_pad; p.rot = rot;
    p.page = page; p.interleaved = interleaved; p.unit_norm = unit_norm; p.max_pos = max_pos; p.eps = eps;
    p.q_w = (const T*)q_w; p.k_w = (const T*)k_w; p.conv_w = (const T*)conv_w; p.ring = (T*)ring;
    p.state_slots = (const int32_t*)state_slots; p.cu_q = (const int32_t*)cu_q; p.kv_lens = (const int32_t*)kv_lens;
    p.n_seqs = n_seqs; p.taps = taps;
    const auto keep = [&] {
      if (taps > 1 && long_portions)
        launch_pdl(conv_keep_kernel<T>, dim3((unsigned)((p.channels() + 255) / 256), n_seqs), dim3(256), 0, s, p);
    };
    if constexpr (sizeof(T) == 2) {
      const auto a16 = [](const void* x) { return (((uintptr_t)x) & 15) == 0; };
      const int tph = d >> 3, hl = rot >> 4;
      if (d % 8 == 0 && dv % 8 == 0 && d <= 256 && (tph & (tph - 1)) == 0 && d_pad % 8 == 0 && ld % 8 == 0 && a16(q) && a16(k) && a16(v) &&
          a16(q_out) && a16(k_cache) && a16(v_cache) && (rot == 0 || (rot % 8 == 0 && a16(cos_sin))) && a16(q_w) && a16(k_w) &&
          (interleaved || rot == 0 || (rot % 16 == 0 && (hl & (hl - 1)) == 0))) {
        if (taps == 0) {
          if (q_w == nullptr && d == dv) launch_pdl(rope_norm_kv_vec_kernel<false, true>, dim3(tokens), block, 0, s, p);
          else if (q_w == nullptr) launch_pdl(rope_norm_kv_vec_kernel<false, false>, dim3(tokens), block, 0, s, p);
          else if (d == dv) launch_pdl(rope_norm_kv_vec_kernel<true, true>, dim3(tokens), block, 0, s, p);
          else launch_pdl(rope_norm_kv_vec_kernel<true, false>, dim3(tokens), block, 0, s, p);
          return;
        }
        if (taps <= kMaxTaps && !unit_norm && !(interleaved && rot > 0) && a16(conv_w) && a16(ring)) {
          const int V = d <= 128 ? 4 : 8, qk = ((nq + nkv) * (d / V) + 255) / 256, parts = qk + (nkv * (dv / V) + 255) / 256;
          const dim3 grid((tokens + kConvRun - 1) / kConvRun, parts), rows(tokens, parts);
          if (V == 4 && long_portions) launch_pdl(conv_rope_kv_kernel<kConvRun, 4>, grid, block, 0, s, p, qk);
          else if (V == 4) launch_pdl(conv_rope_kv_kernel<1, 4>, rows, block, 0, s, p, qk);
          else if (long_portions) launch_pdl(conv_rope_kv_kernel<kConvRun, 8>, grid, block, 0, s, p, qk);
          else launch_pdl(conv_rope_kv_kernel<1, 8>, rows, block, 0, s, p, qk);
          keep();
          return;
        }
      }
    }
    launch_pdl(rope_norm_kv_kernel<T>, grid, block, 0, s, p);
    keep();
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return XLLM_LAUNCH_CHECK();
}

// Convolution (taps >= 1), norms of whole q and k rows with weights [nq * d] and [nkv * d], unit norm of every value head, cache
// write; arguments as above.
XLLM_API int xllm_conv_row_norm_kv(const void* q, const void* k, const void* v, int64_t ld, void* q_out, void* k_cache, void* v_cache,
                                   const void* slots, int tokens, int nq, int nkv, int d, int dv, int d_pad, int page, float eps,
                                   const void* q_w, const void* k_w, const void* conv_w, void* ring, const void* state_slots,
                                   const void* cu_q, const void* kv_lens, int n_seqs, int taps, int long_portions, int dtype,
                                   void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (d <= 0 || dv <= 0 || d_pad < d || d_pad < dv || page <= 0 || nq <= 0 || nkv <= 0 || q_w == nullptr || k_w == nullptr ||
      taps < 1 || conv_w == nullptr || ring == nullptr || state_slots == nullptr || cu_q == nullptr || kv_lens == nullptr || n_seqs <= 0)
    return (int)cudaErrorInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    RopeNormParams<T> p{};
    p.q = (const T*)q; p.k = (const T*)k; p.v = (const T*)v; p.ld = ld; p.q_out = (T*)q_out; p.k_cache = (T*)k_cache;
    p.v_cache = (T*)v_cache; p.slots = (const int32_t*)slots; p.tokens = tokens; p.nq = nq; p.nkv = nkv; p.d = d; p.dv = dv;
    p.d_pad = d_pad; p.page = page; p.eps = eps; p.q_w = (const T*)q_w; p.k_w = (const T*)k_w; p.conv_w = (const T*)conv_w;
    p.ring = (T*)ring; p.state_slots = (const int32_t*)state_slots; p.cu_q = (const int32_t*)cu_q;
    p.kv_lens = (const int32_t*)kv_lens; p.n_seqs = n_seqs; p.taps = taps;
    bool done = false;
    if constexpr (sizeof(T) == 2) {
      const auto a16 = [](const void* x) { return (((uintptr_t)x) & 15) == 0; };
      const int64_t vecs = p.channels() / 8;
      const size_t smem = (size_t)nkv * (dv / 8) * 2 * 4;
      if (d % 8 == 0 && dv % 8 == 0 && d_pad % 8 == 0 && ld % 8 == 0 && taps <= kMaxTaps && vecs <= 3 * kRowThreads && smem <= 32768 &&
          a16(q) && a16(k) && a16(v) && a16(q_out) && a16(k_cache) && a16(v_cache) && a16(q_w) && a16(k_w) && a16(conv_w) && a16(ring)) {
        const bool runs = long_portions && tokens > 4 * 148;
        const dim3 grid(runs ? (tokens + kConvRun - 1) / kConvRun : tokens), block(kRowThreads);
        const auto go = [&](auto many, auto one) { launch_pdl(runs ? many : one, grid, block, smem, s, p, long_portions); };
        if (vecs <= kRowThreads) go(conv_row_norm_kernel<kConvRun, 1>, conv_row_norm_kernel<1, 1>);
        else if (vecs <= 2 * kRowThreads) go(conv_row_norm_kernel<kConvRun, 2>, conv_row_norm_kernel<1, 2>);
        else go(conv_row_norm_kernel<kConvRun, 3>, conv_row_norm_kernel<1, 3>);
        done = true;
      }
    }
    if (!done) launch_pdl(conv_row_norm_any_kernel<T>, dim3(tokens), dim3(256), 0, s, p);
    if (taps > 1 && long_portions) launch_pdl(conv_keep_kernel<T>, dim3((unsigned)((p.channels() + 255) / 256), n_seqs), dim3(256), 0, s, p);
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return XLLM_LAUNCH_CHECK();
}
