// Rotary positions, then a per-head RMS norm without a weight, on q and k of packed projection rows; k goes to
// the paged K cache and the values (any column block of the row: their own projection, or the keys as projected)
// to the V cache.  One pass, any head size up to 512, bf16 or fp32.
//
// The sibling of rope_kv.cu (norm with a weight BEFORE the rotation, power-of-two head sizes).  Heads may be
// stored wider than they are (d_pad >= d, zero filled): the attention kernels take head sizes 64, 128 and 256.
// One warp per (token, head); a lane owns element pairs.
#include "vec_io.cuh"

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
};

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
    float u = to_f32(src[i0]), v = i1 < p.d ? to_f32(src[i1]) : 0.f;
    if (n < half && cs != nullptr) {
      const float c = cs[n], s = cs[half + n];
      const float u2 = u * c - v * s;
      v = v * c + u * s;
      u = u2;
    }
    a[i] = u;
    b[i] = v;
    ss += u * u + v * v;
  }
  float inv = 1.f;
  if (p.unit_norm) inv = 1.f / sqrtf(warp_sum(ss) / (float)p.d + p.eps);
  const int slot = is_q ? 0 : p.slots[t];
  if (!is_q && slot < 0) return;
  const int64_t blk = slot / p.page;
  const int off = slot - (int)blk * p.page;
  const int64_t crow = ((blk * p.nkv + g) * p.page + off) * (int64_t)p.d_pad;
  T* dst = is_q ? p.q_out + (t * p.nq + g) * p.d_pad : p.k_cache + crow;
#pragma unroll
  for (int i = 0; i < kPairs; ++i) {
    const int n = lane + 32 * i;
    if (n >= n_pairs) continue;
    int i0, i1;
    if (n < half && !p.interleaved) { i0 = n; i1 = n + half; }
    else { i0 = 2 * n; i1 = 2 * n + 1; }
    dst[i0] = from_f32<T>(a[i] * inv);
    if (i1 < p.d) dst[i1] = from_f32<T>(b[i] * inv);
  }
  for (int i = p.d + lane; i < p.d_pad; i += 32) dst[i] = from_f32<T>(0.f);
  if (!is_q) {
    const T* vs = p.v + t * p.ld + (int64_t)g * p.dv;
    T* vd = p.v_cache + crow;
    for (int i = lane; i < p.d_pad; i += 32) vd[i] = i < p.dv ? vs[i] : from_f32<T>(0.f);
  }
}

// bf16 heads of 8, 16, ... 256 elements with aligned rows: one CTA per token, a thread owns eight contiguous elements
// of up to four heads, whose 16-byte loads are all issued first (the layout of rope_kv.cu).
constexpr int kVecHeads = 4;

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
      if (!is_q && p.v != p.k)
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
      if (!is_q) *reinterpret_cast<bf16x8*>(p.v_cache + crow + e0) = p.v != p.k ? val[u] : raw[u];
      for (int z = p.d + e0; z < p.d_pad; z += p.d) {
        *reinterpret_cast<uint4*>(dst + z) = make_uint4(0, 0, 0, 0);
        if (!is_q) *reinterpret_cast<uint4*>(p.v_cache + crow + z) = make_uint4(0, 0, 0, 0);
      }
    }
  }
}

}  // namespace xllm

// dtype: 0 bf16, 1 fp32.  rot <= d, rot even.  dv: size of a value head (d where v is the key block).
XLLM_API int xllm_rope_norm_kv(const void* q, const void* k, const void* v, int64_t ld, void* q_out, void* k_cache,
                               void* v_cache, const void* cos_sin, int64_t max_pos, const void* positions, const void* slots,
                               int tokens, int nq, int nkv, int d, int dv, int d_pad, int rot, int page, int interleaved, int unit_norm,
                               float eps, int dtype, void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (d <= 0 || d > 64 * kPairs || d_pad < d || dv <= 0 || d_pad < dv || rot < 0 || rot > d || rot % 2 != 0 || page <= 0 || nq <= 0 || nkv <= 0)
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
    if constexpr (sizeof(T) == 2) {
      const auto a16 = [](const void* x) { return (((uintptr_t)x) & 15) == 0; };
      const int tph = d >> 3, hl = rot >> 4;
      if (d % 8 == 0 && d == dv && d <= 256 && (tph & (tph - 1)) == 0 && d_pad % 8 == 0 && ld % 8 == 0 && a16(q) && a16(k) && a16(v) &&
          a16(q_out) && a16(k_cache) && a16(v_cache) && (rot == 0 || (rot % 8 == 0 && a16(cos_sin))) &&
          (interleaved || rot == 0 || (rot % 16 == 0 && (hl & (hl - 1)) == 0))) {
        launch_pdl(rope_norm_kv_vec_kernel, dim3(tokens), dim3(256), 0, s, p);
        return;
      }
    }
    launch_pdl(rope_norm_kv_kernel<T>, grid, block, 0, s, p);
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return XLLM_LAUNCH_CHECK();
}
