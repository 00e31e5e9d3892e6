// Projections of few outputs whose result stays fp32: router logits, the gates and step sizes of a recurrence.
//
//   out[t, n] = sum_k x[t, k] w[n, k] + b[n]        x, w, b bf16, fp32 sums and result
//
// One CTA per 16 rows x 32 outputs; its eight warps share K (each takes every eighth step of 32) and add up through shared
// memory.  A lane reads eight neighbouring k at a time, of rows and weights alike: a sum does not care in which order its
// terms sit in the operands of the tensor-core product.
#include "attn_common.cuh"
#include "vec_io.cuh"

namespace xllm {

__global__ void __launch_bounds__(256) proj_f32_kernel(float* __restrict__ out, int64_t out_ld, const bf16* __restrict__ x,
                                                       int64_t x_ld, const bf16* __restrict__ w, const bf16* __restrict__ bias,
                                                       int T, int N, int K) {
  __shared__ float part[8][16][33];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * 16, n0 = blockIdx.y * 32, r = lane >> 2, kc = (lane & 3) * 8;
  float c[4][4];
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) c[j][e] = 0.f;
  pdl_wait();
  pdl_launch_dependents();
  const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll 2
  for (int k = warp * 32; k < K; k += 256) {
    const bool on = k + kc < K;                              // K is a multiple of 8
    uint4 a[2], b[4];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = t0 + r + 8 * u;
      a[u] = on && t < T ? *reinterpret_cast<const uint4*>(x + (int64_t)t * x_ld + k + kc) : zero;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + j * 8 + r;
      b[j] = on && n < N ? *reinterpret_cast<const uint4*>(w + (int64_t)n * K + k + kc) : zero;
    }
    const uint32_t a0[4] = {a[0].x, a[1].x, a[0].y, a[1].y}, a1[4] = {a[0].z, a[1].z, a[0].w, a[1].w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      mma_bf16_16816(c[j], a0, b[j].x, b[j].y);
      mma_bf16_16816(c[j], a1, b[j].z, b[j].w);
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) part[warp][r + (e >> 1) * 8][j * 8 + (lane & 3) * 2 + (e & 1)] = c[j][e];
  __syncthreads();
  for (int i = threadIdx.x; i < 512; i += 256) {
    const int t = i >> 5, n = i & 31;
    if (t0 + t >= T || n0 + n >= N) continue;
    float s = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) s += part[q][t][n];
    if (bias != nullptr) s += __bfloat162float(bias[n0 + n]);
    out[(int64_t)(t0 + t) * out_ld + n0 + n] = s;
  }
}

}  // namespace xllm

// x [T, K] with row stride x_ld, w [N, K] dense, bias [N] or null, out fp32 [T, N] with row stride out_ld.
XLLM_API int xllm_proj_f32(void* out, int64_t out_ld, const void* x, int64_t x_ld, const void* w, const void* bias, int T, int N,
                           int K, void* stream) {
  using namespace xllm;
  if (T == 0 || N == 0) return 0;
  if (K <= 0 || K % 8 || x_ld % 8 || (((uintptr_t)x | (uintptr_t)w) & 15)) return (int)cudaErrorInvalidValue;
  launch_pdl(proj_f32_kernel, dim3((T + 15) / 16, (N + 31) / 32), dim3(256), 0, (cudaStream_t)stream, (float*)out, out_ld,
             (const bf16*)x, x_ld, (const bf16*)w, (const bf16*)bias, T, N, K);
  return XLLM_LAUNCH_CHECK();
}
