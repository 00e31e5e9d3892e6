// Finishes the raw fp32 head outputs of a recurrence, and gates attention outputs:
//
//   out[t, h dv + i] = o[t, h, i] / div[t, h] / rms over the head * w * act(g[t, h dv + i])       head_norm_gate
//   out[t, h dv + i] = a[t, h, i] * sigmoid(g[t, h dv + i])   or sigmoid(g[t, h])                    head_gate
//
// every factor optional in the first (a head may be a whole row; w: one weight per element shared by the heads, or one per head and element; act:
// silu or sigmoid).  The heads of `a` may be stored wider than dv.  A warp owns whole heads.
#include "vec_io.cuh"

namespace xllm {

template <typename T>
struct HeadNormParams {
  T* out;
  const float* o;        // [T, H, dv]
  const float* div;      // [T, H] or null
  const T* g;            // row stride g_ld, or null
  const T* w;            // element i of head h at h * w_head + i, or null
  int64_t out_ld, g_ld, items;
  int H, dv, w_head, unit_norm, act;
  float eps;
};

template <typename T>
__device__ __forceinline__ float gate_act(float z, int act) {
  const float s = sigmoid_as<T>(z);
  return act == 0 ? z * s : s;
}

// heads of up to 128 elements, four at a time: a warp owns U neighbouring items whose loads are all in flight together
template <typename T, int U>
__global__ void __launch_bounds__(256) head_norm_gate_small_kernel(HeadNormParams<T> p) {
  const int lane = threadIdx.x & 31, c = lane * 4;
  const int64_t first = ((int64_t)blockIdx.x * 8 + (threadIdx.x >> 5)) * U;
  const bool on = c < p.dv;
  pdl_wait();
  pdl_launch_dependents();
  float x[U][4], z[U][4], f[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int64_t it = first + u;
    f[u] = 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) x[u][j] = z[u][j] = 0.f;
    if (it >= p.items) continue;
    const unsigned t = (unsigned)it / (unsigned)p.H;         // fewer than 2^32 items
    const int h = (int)((unsigned)it - t * p.H);
    if (on) load_f32<4>(p.o + it * p.dv + c, x[u]);
    if (on && p.g != nullptr) load_f32<4>(p.g + t * p.g_ld + (int64_t)h * p.dv + c, z[u]);
    if (p.div != nullptr) f[u] = p.div[it];
  }
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int64_t it = first + u;
    if (it >= p.items) break;
    const unsigned t = (unsigned)it / (unsigned)p.H;
    const int h = (int)((unsigned)it - t * p.H);
    const float s = f[u] > 0.f ? 1.f / f[u] : 0.f;               // rows of no sequence have no denominator
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      x[u][j] *= s;
      ss += x[u][j] * x[u][j];
    }
    const float inv = p.unit_norm ? 1.f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps) : 1.f;
    if (!on) continue;
    float w[4];
    if (p.w != nullptr) {
      load_f32<4>(p.w + (int64_t)h * p.w_head + c, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) x[u][j] *= w[j];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      x[u][j] *= inv;
      if (p.g != nullptr) x[u][j] *= gate_act<T>(z[u][j], p.act);
    }
    store_f32<4>(p.out + t * p.out_ld + (int64_t)h * p.dv + c, x[u]);
  }
}

// V elements per lane and step; with V = 4 a head of up to 512 elements stays in registers
template <typename T, int V>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(HeadNormParams<T> p) {
  constexpr int NI = 4;
  const int lane = threadIdx.x & 31;
  const int64_t it = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  pdl_wait();
  pdl_launch_dependents();
  if (it >= p.items) return;
  const int64_t t = it / p.H;
  const int h = (int)(it - t * p.H);
  const float* src = p.o + it * p.dv;
  float f = 1.f;
  if (p.div != nullptr) {
    const float d = p.div[it];
    f = d > 0.f ? 1.f / d : 0.f;             // rows of no sequence have no denominator
  }
  float x[NI][V];
  float ss = 0.f;
  for (int c0 = 0; c0 < p.dv; c0 += 32 * V * NI) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = c0 + (lane + 32 * i) * V;
      if (c >= p.dv) continue;
      load_f32<V>(src + c, x[i]);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        x[i][j] *= f;
        ss += x[i][j] * x[i][j];
      }
    }
  }
  float inv = 1.f;
  if (p.unit_norm) inv = 1.f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
  T* dst = p.out + t * p.out_ld + (int64_t)h * p.dv;
  const T* gr = p.g != nullptr ? p.g + t * p.g_ld + (int64_t)h * p.dv : nullptr;
  const T* w = p.w != nullptr ? p.w + (int64_t)h * p.w_head : nullptr;
  for (int c0 = 0; c0 < p.dv; c0 += 32 * V * NI) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = c0 + (lane + 32 * i) * V;
      if (c >= p.dv) continue;
      if (p.dv > 32 * V * NI) {              // does not fit the registers: read again
        load_f32<V>(src + c, x[i]);
#pragma unroll
        for (int j = 0; j < V; ++j) x[i][j] *= f;
      }
      float y[V], u[V];
#pragma unroll
      for (int j = 0; j < V; ++j) y[j] = x[i][j] * inv;
      if (w != nullptr) {
        load_f32<V>(w + c, u);
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] *= u[j];
      }
      if (gr != nullptr) {
        load_f32<V>(gr + c, u);
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] *= gate_act<T>(u[j], p.act);
      }
      store_f32<V>(dst + c, y);
    }
  }
}

// one item per CTA: heads (whole rows, where all heads are normed together) too large for a warp
template <typename T, int V>
__global__ void __launch_bounds__(256) row_norm_gate_kernel(HeadNormParams<T> p) {
  constexpr int NI = 4;
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t it = blockIdx.x, t = it / p.H;
  const int h = (int)(it - t * p.H);
  const float* src = p.o + it * p.dv;
  float f = 1.f;
  if (p.div != nullptr) {
    const float d = p.div[it];
    f = d > 0.f ? 1.f / d : 0.f;
  }
  float x[NI][V];
  float ss = 0.f;
  for (int c0 = 0; c0 < p.dv; c0 += 256 * V * NI) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = c0 + (threadIdx.x + 256 * i) * V;
      if (c >= p.dv) continue;
      load_f32<V>(src + c, x[i]);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        x[i][j] *= f;
        ss += x[i][j] * x[i][j];
      }
    }
  }
  float inv = 1.f;
  if (p.unit_norm) inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.dv + p.eps);
  T* dst = p.out + t * p.out_ld + (int64_t)h * p.dv;
  const T* gr = p.g != nullptr ? p.g + t * p.g_ld + (int64_t)h * p.dv : nullptr;
  const T* w = p.w != nullptr ? p.w + (int64_t)h * p.w_head : nullptr;
  for (int c0 = 0; c0 < p.dv; c0 += 256 * V * NI) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = c0 + (threadIdx.x + 256 * i) * V;
      if (c >= p.dv) continue;
      if (p.dv > 256 * V * NI) {             // does not fit the registers: read again
        load_f32<V>(src + c, x[i]);
#pragma unroll
        for (int j = 0; j < V; ++j) x[i][j] *= f;
      }
      float y[V], u[V];
#pragma unroll
      for (int j = 0; j < V; ++j) y[j] = x[i][j] * inv;
      if (w != nullptr) {
        load_f32<V>(w + c, u);
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] *= u[j];
      }
      if (gr != nullptr) {
        load_f32<V>(gr + c, u);
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] *= gate_act<T>(u[j], p.act);
      }
      store_f32<V>(dst + c, y);
    }
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) head_gate_kernel(T* __restrict__ out, const T* __restrict__ a, const T* __restrict__ g,
                                                        int64_t g_ld, int64_t tokens, int H, int dv, int d_pad,
                                                        int per_head) {
  pdl_wait();
  pdl_launch_dependents();
  const int per = dv / V, row = H * per;
  for (int64_t n = blockIdx.x * (int64_t)256 + threadIdx.x; n < tokens * row; n += (int64_t)gridDim.x * 256) {
    const int64_t t = n < (1LL << 32) ? (unsigned)n / (unsigned)row : n / row;
    const int r = (int)(n - t * row), h = r / per, i = (r - h * per) * V;
    float x[V], z[V];
    load_f32<V>(a + (t * H + h) * d_pad + i, x);
    if (per_head) {
      const float f = gate_act<T>(to_f32(g[t * g_ld + h]), 1);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= f;
      store_f32<V>(out + (t * H + h) * (int64_t)dv + i, x);
      continue;
    }
    load_f32<V>(g + t * g_ld + (int64_t)h * dv + i, z);
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] *= gate_act<T>(z[j], 1);
    store_f32<V>(out + (t * H + h) * (int64_t)dv + i, x);
  }
}

}  // namespace xllm

// dtype: 0 bf16, 1 fp32 (out, g, w).  act: 0 silu, 1 sigmoid.
XLLM_API int xllm_head_norm_gate(void* out, int64_t out_ld, const void* o, const void* div, const void* g, int64_t g_ld,
                                 const void* w, int w_head, int64_t tokens, int H, int dv, int unit_norm, int act, float eps,
                                 int dtype, void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (H <= 0 || dv <= 0 || act < 0 || act > 1) return (int)cudaErrorInvalidValue;
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    HeadNormParams<T> p{(T*)out, (const float*)o, (const float*)div, (const T*)g, (const T*)w, out_ld, g_ld, tokens * H, H, dv,
                        w_head, unit_norm, act, eps};
    const auto al = [](const void* x, size_t a) { return (((uintptr_t)x) & (a - 1)) == 0; };
    const size_t v = 4 * sizeof(T);
    const dim3 grid((unsigned)((p.items + 7) / 8)), block(256);
    if (dv % 4 == 0 && out_ld % 4 == 0 && (g == nullptr || g_ld % 4 == 0) && w_head % 4 == 0 && al(out, v) && al(o, 16) &&
        al(g, v) && al(w, v) && dv <= 128 && p.items < (1LL << 32))
      launch_pdl(head_norm_gate_small_kernel<T, 4>, dim3((unsigned)((p.items + 31) / 32)), block, 0, (cudaStream_t)stream, p);
    else if (dv > 512 && p.items < (1LL << 31)) {
      const dim3 rows((unsigned)p.items);
      if (dv % 4 == 0 && out_ld % 4 == 0 && (g == nullptr || g_ld % 4 == 0) && w_head % 4 == 0 && al(out, v) && al(o, 16) &&
          al(g, v) && al(w, v))
        launch_pdl(row_norm_gate_kernel<T, 4>, rows, block, 0, (cudaStream_t)stream, p);
      else
        launch_pdl(row_norm_gate_kernel<T, 1>, rows, block, 0, (cudaStream_t)stream, p);
    } else if (dv % 4 == 0 && out_ld % 4 == 0 && (g == nullptr || g_ld % 4 == 0) && w_head % 4 == 0 && al(out, v) && al(o, 16) &&
             al(g, v) && al(w, v))
      launch_pdl(head_norm_gate_kernel<T, 4>, grid, block, 0, (cudaStream_t)stream, p);
    else
      launch_pdl(head_norm_gate_kernel<T, 1>, grid, block, 0, (cudaStream_t)stream, p);
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return XLLM_LAUNCH_CHECK();
}

// a [tokens, H, d_pad] -> out [tokens, H * dv] times the sigmoid of g [tokens, H * dv] or (per_head) [tokens, H], row stride g_ld
XLLM_API int xllm_head_gate(void* out, const void* a, const void* g, int64_t g_ld, int64_t tokens, int H, int dv, int d_pad,
                            int per_head, int dtype, void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (H <= 0 || dv <= 0 || d_pad < dv) return (int)cudaErrorInvalidValue;
  const auto al = [](const void* x) { return (((uintptr_t)x) & 15) == 0; };
  const bool v8 = dv % 8 == 0 && d_pad % 8 == 0 && al(out) && al(a) && (per_head || (g_ld % 8 == 0 && al(g)));
  const int64_t want = (tokens * H * (v8 ? dv / 8 : dv) + 255) / 256;
  const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16));
  const auto run = [&](auto tag) {
    using T = decltype(tag);
    if (v8)
      launch_pdl(head_gate_kernel<T, 8>, grid, dim3(256), 0, (cudaStream_t)stream, (T*)out, (const T*)a, (const T*)g, g_ld,
                 tokens, H, dv, d_pad, per_head);
    else
      launch_pdl(head_gate_kernel<T, 1>, grid, dim3(256), 0, (cudaStream_t)stream, (T*)out, (const T*)a, (const T*)g, g_ld,
                 tokens, H, dv, d_pad, per_head);
  };
  if (dtype == 0) run(bf16());
  else run(float());
  return XLLM_LAUNCH_CHECK();
}
