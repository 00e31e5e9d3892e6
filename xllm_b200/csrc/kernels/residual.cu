// An fp32 residual stream: branch outputs join it and the next sublayer's input leaves it in one pass.
//
//   x[t] = (init ? 0 : x[t]) + n(coef * sum_i n_i(y_i[t]))     n_i: identity, or RMS norm with a weight; n likewise
//   out[t] = rmsnorm(x[t]) * (w + offset)   or   cast(x[t])       offset: 1 for weights stored around zero
//
// One launch covers: the embedding (init, y_0 gathered by token id) + first norm; a plain branch + the
// next norm; a branch that is normalised before it joins (post-norm) + the next norm; two branches that
// are normalised and averaged; and the un-normalised cast that a projection of the residual itself reads.
// A row lives in the registers of a group of TPR threads; the group size depends on the width only, so a
// row is reduced in the same order whatever batch it arrives in.  No counterpart in the reference, whose
// residual stream is bf16 (xllm/core/kernels/cuda/norm.cu:43-174).
//
// Norm after the sum (a stream that is itself normed, in `groups` consecutive parts of its own mean square each):
//
//   x[t] = norm(alpha * x[t] + y[t]) * w;   out[t] = cast(x[t])   or   norm(x[t]) * w_out
//
// A part depends on nothing outside it, so the kernel takes every part as a row.
//
// Also here: the token-indexed gated activation of a per-token side input, and the fp32 form of the gated
// activation of a dense MLP.
#include "vec_io.cuh"

namespace xllm {

struct ResidualParams {
  float* x;               // [T, hidden] fp32, dense
  const void* y[2];       // branches, row stride y_ld[i] elements
  const void* w[2];       // norm weight of branch i, or null
  const void* w_sum;      // norm weight of the branches' sum, or null
  const int64_t* rows;    // y[0] row of token t is rows[t] (embedding), or null
  const void* w_out;      // norm weight of the output, or null: cast
  void* out;              // [T, hidden] dense, or null
  int64_t y_ld[2];
  int64_t n_rows;         // rows of the gathered table
  int tokens, hidden, init;
  float coef, eps, w_out_offset;   // the output's norm weight is w_out + w_out_offset
};

constexpr int kResVec = 4;   // vectors per thread

template <int TPR>
__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  if constexpr (TPR > 32) {
    constexpr int W = TPR / 32;
    const int wid = threadIdx.x >> 5;
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[wid] = v;
    __syncthreads();
    const int g = wid / W * W;
    v = 0.f;
#pragma unroll
    for (int i = 0; i < W; ++i) v += red[g + i];
  }
  return v;
}

template <typename T, int V, int TPR, int NB, bool NORM_SUM>
__global__ void __launch_bounds__(TPR > 256 ? TPR : 256) residual_kernel(ResidualParams p) {
  __shared__ float red[32];
  const int t = threadIdx.x % TPR;
  const int64_t row = (int64_t)blockIdx.x * (blockDim.x / TPR) + threadIdx.x / TPR;
  const bool live = row < p.tokens;
  const int nvec = p.hidden / V;
  pdl_wait();
  pdl_launch_dependents();
  float acc[kResVec][V];
  float br[NB][kResVec][V];
  const T* yr[NB];
#pragma unroll
  for (int b = 0; b < NB; ++b) {
    int64_t r = row;
    if (b == 0 && p.rows != nullptr && live) {
      r = p.rows[row];
      r = r < 0 ? 0 : (r >= p.n_rows ? p.n_rows - 1 : r);
    }
    yr[b] = reinterpret_cast<const T*>(p.y[b]) + r * p.y_ld[b];
  }
  float* xr = p.x + row * p.hidden;
#pragma unroll
  for (int i = 0; i < kResVec; ++i) {
    const int v = t + i * TPR;
    const bool on = live && v < nvec;
#pragma unroll
    for (int j = 0; j < V; ++j) acc[i][j] = 0.f;
    if (on && !p.init) load_f32<V>(xr + v * V, acc[i]);
#pragma unroll
    for (int b = 0; b < NB; ++b) {
#pragma unroll
      for (int j = 0; j < V; ++j) br[b][i][j] = 0.f;
      if (on) load_f32<V>(yr[b] + v * V, br[b][i]);
    }
  }
#pragma unroll
  for (int b = 0; b < NB; ++b) {
    float inv = p.coef;
    if (p.w[b] != nullptr) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < kResVec; ++i)
#pragma unroll
        for (int j = 0; j < V; ++j) ss += br[b][i][j] * br[b][i][j];
      ss = row_sum<TPR>(ss, red);
      inv = p.coef / sqrtf(ss / (float)p.hidden + p.eps);
    }
#pragma unroll
    for (int i = 0; i < kResVec; ++i) {
      const int v = t + i * TPR;
      if (!(live && v < nvec)) continue;
      float w[V];
      if (p.w[b] != nullptr) {
        load_f32<V>(reinterpret_cast<const T*>(p.w[b]) + v * V, w);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) w[j] = 1.f;
      }
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float z = br[b][i][j] * inv * w[j];
        if (!NORM_SUM) acc[i][j] += z;
        else if (b == 0) br[0][i][j] = z;
        else br[0][i][j] += z;
      }
    }
  }
  if constexpr (NORM_SUM) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kResVec; ++i)
#pragma unroll
      for (int j = 0; j < V; ++j) ss += br[0][i][j] * br[0][i][j];
    const float inv = 1.f / sqrtf(row_sum<TPR>(ss, red) / (float)p.hidden + p.eps);
#pragma unroll
    for (int i = 0; i < kResVec; ++i) {
      const int v = t + i * TPR;
      if (!(live && v < nvec)) continue;
      float w[V];
      load_f32<V>(reinterpret_cast<const T*>(p.w_sum) + v * V, w);
#pragma unroll
      for (int j = 0; j < V; ++j) acc[i][j] += br[0][i][j] * inv * w[j];
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kResVec; ++i) {
    const int v = t + i * TPR;
    if (live && v < nvec) store_f32<V>(xr + v * V, acc[i]);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += acc[i][j] * acc[i][j];
  }
  if (p.out == nullptr) return;
  float inv = 1.f;
  if (p.w_out != nullptr) {
    ss = row_sum<TPR>(ss, red);
    inv = 1.f / sqrtf(ss / (float)p.hidden + p.eps);
  }
  T* orow = reinterpret_cast<T*>(p.out) + row * p.hidden;
#pragma unroll
  for (int i = 0; i < kResVec; ++i) {
    const int v = t + i * TPR;
    if (!(live && v < nvec)) continue;
    float o[V];
    if (p.w_out != nullptr) {
      float w[V];
      load_f32<V>(reinterpret_cast<const T*>(p.w_out) + v * V, w);
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] = acc[i][j] * inv * (w[j] + p.w_out_offset);
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] = acc[i][j];
    }
    store_f32<V>(orow + v * V, o);
  }
}

template <typename T, int V, int NB, bool NORM_SUM = false>
static int launch_residual(const ResidualParams& p, cudaStream_t s) {
  const int nvec = p.hidden / V;
  int tpr = 32;
  while (tpr < 1024 && nvec > tpr * kResVec) tpr <<= 1;
  if (nvec > tpr * kResVec) return (int)cudaErrorInvalidValue;
  const int block = tpr > 256 ? tpr : 256;
  const int rows = block / tpr;
  const dim3 grid((unsigned)((p.tokens + rows - 1) / rows));
#define XLLM_RES_CASE(N)                                                              \
  case N:                                                                             \
    launch_pdl(residual_kernel<T, V, N, NB, NORM_SUM>, grid, dim3(block), 0, s, p);             \
    break;
  switch (tpr) {
    XLLM_RES_CASE(32)
    XLLM_RES_CASE(64)
    XLLM_RES_CASE(128)
    XLLM_RES_CASE(256)
    XLLM_RES_CASE(512)
    XLLM_RES_CASE(1024)
  }
#undef XLLM_RES_CASE
  return XLLM_LAUNCH_CHECK();
}

struct PostNormParams {
  float* x;               // [T, hidden] fp32, dense
  const void* y;          // row stride y_ld
  const void *w, *w_out;  // [hidden]; w_out null: cast
  void* out;              // [T, hidden] dense
  int64_t y_ld, rows;     // rows: tokens * groups
  int hidden, groups, part;
  float alpha, eps;
};

template <typename T, int V, int TPR>
__global__ void __launch_bounds__(TPR > 256 ? TPR : 256) postnorm_kernel(PostNormParams p) {
  __shared__ float red[32];
  const int t = threadIdx.x % TPR;
  const int64_t row = (int64_t)blockIdx.x * (blockDim.x / TPR) + threadIdx.x / TPR;
  const bool live = row < p.rows;
  const int64_t tok = live ? row / p.groups : 0;
  const int col = live ? (int)(row - tok * p.groups) * p.part : 0;
  const int nvec = p.part / V;
  pdl_wait();
  pdl_launch_dependents();
  float* xr = p.x + tok * p.hidden + col;
  const T* yr = reinterpret_cast<const T*>(p.y) + tok * p.y_ld + col;
  float acc[kResVec][V], br[kResVec][V];
#pragma unroll
  for (int i = 0; i < kResVec; ++i) {
    const int v = t + i * TPR;
#pragma unroll
    for (int j = 0; j < V; ++j) acc[i][j] = br[i][j] = 0.f;
    if (live && v < nvec) {
      load_f32<V>(xr + v * V, acc[i]);
      load_f32<V>(yr + v * V, br[i]);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kResVec; ++i)
#pragma unroll
    for (int j = 0; j < V; ++j) {
      acc[i][j] = fmaf(p.alpha, acc[i][j], br[i][j]);
      ss += acc[i][j] * acc[i][j];
    }
  float inv = 1.f / sqrtf(row_sum<TPR>(ss, red) / (float)p.part + p.eps);
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kResVec; ++i) {
    const int v = t + i * TPR;
    if (!(live && v < nvec)) continue;
    float w[V];
    load_f32<V>(reinterpret_cast<const T*>(p.w) + col + v * V, w);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      acc[i][j] *= inv * w[j];
      ss += acc[i][j] * acc[i][j];
    }
    store_f32<V>(xr + v * V, acc[i]);
  }
  if (p.w_out != nullptr) inv = 1.f / sqrtf(row_sum<TPR>(ss, red) / (float)p.part + p.eps);
  T* orow = reinterpret_cast<T*>(p.out) + tok * p.hidden + col;
#pragma unroll
  for (int i = 0; i < kResVec; ++i) {
    const int v = t + i * TPR;
    if (!(live && v < nvec)) continue;
    if (p.w_out != nullptr) {
      float w[V];
      load_f32<V>(reinterpret_cast<const T*>(p.w_out) + col + v * V, w);
#pragma unroll
      for (int j = 0; j < V; ++j) acc[i][j] *= inv * w[j];
    }
    store_f32<V>(orow + v * V, acc[i]);
  }
}

template <typename T, int V>
static int launch_postnorm(const PostNormParams& p, cudaStream_t s) {
  const int nvec = p.part / V;
  int tpr = 32;
  while (tpr < 1024 && nvec > tpr * kResVec) tpr <<= 1;
  if (nvec > tpr * kResVec) return (int)cudaErrorInvalidValue;
  const int block = tpr > 256 ? tpr : 256;
  const int rows = block / tpr;
  const dim3 grid((unsigned)((p.rows + rows - 1) / rows));
#define XLLM_POST_CASE(N)                                                  \
  case N:                                                                  \
    launch_pdl(postnorm_kernel<T, V, N>, grid, dim3(block), 0, s, p);      \
    break;
  switch (tpr) {
    XLLM_POST_CASE(32)
    XLLM_POST_CASE(64)
    XLLM_POST_CASE(128)
    XLLM_POST_CASE(256)
    XLLM_POST_CASE(512)
    XLLM_POST_CASE(1024)
  }
#undef XLLM_POST_CASE
  return XLLM_LAUNCH_CHECK();
}

// out[t, i] = gelu_tanh(gate[t, i]) * table[ids[t], col0 + i] for i < dim, 0 for dim <= i < dim_pad; V columns a thread.
template <typename T, int V>
__global__ void __launch_bounds__(256) gelu_mul_rows_kernel(T* __restrict__ out, const T* __restrict__ gate, int64_t gate_ld,
                                                            const T* __restrict__ table, int64_t table_ld, int64_t n_rows,
                                                            const int64_t* __restrict__ ids, int64_t col0, int tokens, int dim,
                                                            int dim_pad) {
  pdl_wait();
  pdl_launch_dependents();
  const int per = dim_pad / V;
  const int64_t total = (int64_t)tokens * per;
  for (int64_t n = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; n < total; n += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = n / per;
    const int i = (int)(n - t * per) * V;
    float r[V];
#pragma unroll
    for (int j = 0; j < V; ++j) r[j] = 0.f;
    if (i < dim) {                                   // V divides dim, or V = 1
      int64_t id = ids[t];
      id = id < 0 ? 0 : (id >= n_rows ? n_rows - 1 : id);
      float z[V], e[V];
      load_f32<V>(gate + t * gate_ld + i, z);
      load_f32<V>(table + id * table_ld + col0 + i, e);
      const float k = 0.79788456080286535588f;       // sqrt(2 / pi)
#pragma unroll
      for (int j = 0; j < V; ++j)
        r[j] = 0.5f * z[j] * (1.f + tanhf(k * (z[j] + 0.044715f * z[j] * z[j] * z[j]))) * e[j];
    }
    store_f32<V>(out + t * dim_pad + i, r);
  }
}

// out[t, i] = act(x[t, i]) * x[t, d + i], fp32; act: 0 silu, 2 gelu (tanh form), 3 clamped_glu
__global__ void __launch_bounds__(256) act_mul_f32_kernel(float* __restrict__ out, const float* __restrict__ x, int64_t tokens,
                                                          int d, int64_t x_ld, int act, float limit, float alpha) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t total = tokens * d;
  for (int64_t n = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; n < total; n += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = n / d;
    const int i = (int)(n - t * d);
    float z = x[t * x_ld + i], u = x[t * x_ld + d + i];
    if (act == 2) {
      out[n] = 0.5f * z * (1.f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z))) * u;
    } else if (act == 3) {
      z = fminf(z, limit);
      out[n] = z / (1.f + expf(-alpha * z)) * (fminf(fmaxf(u, -limit), limit) + 1.f);
    } else {
      out[n] = z / (1.f + expf(-z)) * u;
    }
  }
}

}  // namespace xllm

// dtype: 0 bf16, 1 fp32 (branches, weights, out).  y1 / w0 / w1 / w_sum / rows / w_out / out may be null.
XLLM_API int xllm_residual_update(void* x, const void* y0, int64_t y0_ld, const void* w0, const void* y1, int64_t y1_ld,
                                  const void* w1, const void* w_sum, const void* rows, int64_t n_rows, const void* w_out, void* out, int tokens,
                                  int hidden, int init, float coef, float eps, float w_out_offset, int dtype,
                                  void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (hidden <= 0 || y0 == nullptr || x == nullptr) return (int)cudaErrorInvalidValue;
  ResidualParams p;
  p.x = (float*)x; p.y[0] = y0; p.y[1] = y1; p.w[0] = w0; p.w[1] = w1; p.w_sum = w_sum; p.rows = (const int64_t*)rows;
  p.w_out = w_out; p.out = out; p.y_ld[0] = y0_ld; p.y_ld[1] = y1_ld; p.n_rows = n_rows; p.tokens = tokens;
  p.hidden = hidden; p.init = init; p.coef = coef; p.eps = eps; p.w_out_offset = w_out_offset;
  const auto a16 = [](const void* q) { return (((uintptr_t)q) & 15) == 0; };
  const bool al = a16(x) && a16(y0) && a16(w0) && a16(y1) && a16(w1) && a16(w_sum) && a16(w_out) && a16(out);
  cudaStream_t s = (cudaStream_t)stream;
  const bool v8 = al && hidden % 8 == 0 && y0_ld % 8 == 0 && y1_ld % 8 == 0;
  if (w_sum != nullptr) {
    if (dtype == 0) {
      if (v8) return y1 ? launch_residual<bf16, 8, 2, true>(p, s) : launch_residual<bf16, 8, 1, true>(p, s);
      return y1 ? launch_residual<bf16, 1, 2, true>(p, s) : launch_residual<bf16, 1, 1, true>(p, s);
    }
    if (v8) return y1 ? launch_residual<float, 8, 2, true>(p, s) : launch_residual<float, 8, 1, true>(p, s);
    return y1 ? launch_residual<float, 1, 2, true>(p, s) : launch_residual<float, 1, 1, true>(p, s);
  }
  if (dtype == 0) {
    if (v8) return y1 ? launch_residual<bf16, 8, 2>(p, s) : launch_residual<bf16, 8, 1>(p, s);
    return y1 ? launch_residual<bf16, 1, 2>(p, s) : launch_residual<bf16, 1, 1>(p, s);
  }
  if (v8) return y1 ? launch_residual<float, 8, 2>(p, s) : launch_residual<float, 8, 1>(p, s);
  return y1 ? launch_residual<float, 1, 2>(p, s) : launch_residual<float, 1, 1>(p, s);
}

XLLM_API int xllm_gelu_mul_rows(void* out, const void* gate, int64_t gate_ld, const void* table, int64_t table_ld,
                                int64_t n_rows, const void* ids, int64_t col0, int tokens, int dim, int dim_pad, int dtype,
                                void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (dim <= 0 || dim_pad < dim || col0 < 0 || col0 + dim > table_ld) return (int)cudaErrorInvalidValue;
  const auto a16 = [](const void* q) { return (((uintptr_t)q) & 15) == 0; };
  const bool v8 = dim % 8 == 0 && dim_pad % 8 == 0 && gate_ld % 8 == 0 && table_ld % 8 == 0 && col0 % 8 == 0 && a16(out) &&
                  a16(gate) && a16(table);
  const int64_t want = ((int64_t)tokens * (v8 ? dim_pad / 8 : dim_pad) + 255) / 256;
  const dim3 grid((unsigned)(want < 148 * 8 ? want : 148 * 8));
  cudaStream_t s = (cudaStream_t)stream;
  const auto run = [&](auto tag, auto kernel) {
    using T = decltype(tag);
    launch_pdl(kernel, grid, dim3(256), 0, s, (T*)out, (const T*)gate, gate_ld, (const T*)table, table_ld, n_rows,
               (const int64_t*)ids, col0, tokens, dim, dim_pad);
  };
  if (dtype == 0) {
    if (v8) run(bf16(), gelu_mul_rows_kernel<bf16, 8>);
    else run(bf16(), gelu_mul_rows_kernel<bf16, 1>);
  } else {
    if (v8) run(float(), gelu_mul_rows_kernel<float, 8>);
    else run(float(), gelu_mul_rows_kernel<float, 1>);
  }
  return XLLM_LAUNCH_CHECK();
}

// act: 0 silu, 2 gelu (tanh form), 3 clamped_glu with `limit` and `alpha`.
XLLM_API int xllm_act_mul_f32(void* out, const void* x, int64_t tokens, int d, int64_t x_ld, int act, float limit, float alpha,
                              void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (act != 0 && act != 2 && act != 3) return (int)cudaErrorInvalidValue;
  const int64_t want = (tokens * d + 255) / 256;
  launch_pdl(act_mul_f32_kernel, dim3((unsigned)(want < 148 * 8 ? want : 148 * 8)), dim3(256), 0, (cudaStream_t)stream,
             (float*)out, (const float*)x, tokens, d, x_ld, act, limit, alpha);
  return XLLM_LAUNCH_CHECK();
}

// x [tokens, hidden] fp32 <- norm(alpha x + y) * w in `groups` parts; out [tokens, hidden] the stream cast or normed with w_out.
// dtype: 0 bf16, 1 fp32 (y, w, w_out, out).
XLLM_API int xllm_postnorm_update(void* x, const void* y, int64_t y_ld, const void* w, const void* w_out, void* out, int64_t tokens,
                                  int hidden, int groups, float alpha, float eps, int dtype, void* stream) {
  using namespace xllm;
  if (tokens == 0) return 0;
  if (hidden <= 0 || groups <= 0 || hidden % groups != 0 || x == nullptr || y == nullptr || w == nullptr || out == nullptr)
    return (int)cudaErrorInvalidValue;
  PostNormParams p{(float*)x, y, w, w_out, out, y_ld, tokens * groups, hidden, groups, hidden / groups, alpha, eps};
  const auto a16 = [](const void* q) { return (((uintptr_t)q) & 15) == 0; };
  const bool v8 = p.part % 8 == 0 && y_ld % 8 == 0 && a16(x) && a16(y) && a16(w) && a16(w_out) && a16(out);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == 0) return v8 ? launch_postnorm<bf16, 8>(p, s) : launch_postnorm<bf16, 1>(p, s);
  return v8 ? launch_postnorm<float, 8>(p, s) : launch_postnorm<float, 1>(p, s);
}
