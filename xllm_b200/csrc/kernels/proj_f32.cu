// Projections of few outputs whose result stays fp32: router logits, the gates and step sizes of a recurrence.
//
//   out[t, n] = sum_k x[t, k] w[n, k] + b[n]        x, w, b bf16, fp32 sums and result
//
// One CTA per 16 or 32 rows x 32 outputs; its sixteen warps share K (each takes every sixteenth step of 32) and add up
// through shared memory.  A lane reads eight neighbouring k at a time, of rows and weights alike: a sum does not care in
// which order its terms sit in the operands of the tensor-core product.
#include "attn_common.cuh"
#include "vec_io.cuh"

namespace xllm {

constexpr int kProjWarps = 16;

// MT: tiles of 16 rows per CTA;  AHEAD: steps whose loads are in flight together
template <int MT, int AHEAD>
__global__ void __launch_bounds__(32 * kProjWarps) proj_f32_kernel(float* __restrict__ out, int64_t out_ld, const bf16* __restrict__ x,
                                                       int64_t x_ld, const bf16* __restrict__ w, const bf16* __restrict__ bias,
                                                       int T, int N, int K) {
  extern __shared__ float part[];                            // [warps][16 MT][33]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * 16 * MT, n0 = blockIdx.y * 32, r = lane >> 2, kc = (lane & 3) * 8;
  float c[MT][4][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) c[i][j][e] = 0.f;
  pdl_wait();
  pdl_launch_dependents();
  const uint4 zero = make_uint4(0, 0, 0, 0);
  const bf16* xp[2 * MT];
  const bf16* wp[4];
#pragma unroll
  for (int u = 0; u < 2 * MT; ++u) xp[u] = t0 + r + 8 * u < T ? x + (int64_t)(t0 + r + 8 * u) * x_ld + kc : nullptr;
#pragma unroll
  for (int j = 0; j < 4; ++j) wp[j] = n0 + j * 8 + r < N ? w + (int64_t)(n0 + j * 8 + r) * K + kc : nullptr;
  for (int k0 = warp * 32; k0 < K; k0 += 32 * kProjWarps * AHEAD) {
    uint4 a[AHEAD][2 * MT], b[AHEAD][4];
#pragma unroll
    for (int s = 0; s < AHEAD; ++s) {
      const int k = k0 + s * 32 * kProjWarps;
      const bool on = k + kc < K;                            // K is a multiple of 8
#pragma unroll
      for (int u = 0; u < 2 * MT; ++u) a[s][u] = on && xp[u] != nullptr ? *reinterpret_cast<const uint4*>(xp[u] + k) : zero;
#pragma unroll
      for (int j = 0; j < 4; ++j) b[s][j] = on && wp[j] != nullptr ? *reinterpret_cast<const uint4*>(wp[j] + k) : zero;
    }
#pragma unroll
    for (int s = 0; s < AHEAD; ++s)
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const uint4 p = a[s][2 * i], q = a[s][2 * i + 1];
        const uint32_t a0[4] = {p.x, q.x, p.y, q.y}, a1[4] = {p.z, q.z, p.w, q.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          mma_bf16_16816(c[i][j], a0, b[s][j].x, b[s][j].y);
          mma_bf16_16816(c[i][j], a1, b[s][j].z, b[s][j].w);
        }
      }
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        part[(warp * 16 * MT + i * 16 + r + (e >> 1) * 8) * 33 + j * 8 + (lane & 3) * 2 + (e & 1)] = c[i][j][e];
  __syncthreads();
  for (int i = threadIdx.x; i < 512 * MT; i += 32 * kProjWarps) {
    const int t = i >> 5, n = i & 31;
    if (t0 + t >= T || n0 + n >= N) continue;
    float s = 0.f;
#pragma unroll
    for (int q = 0; q < kProjWarps; ++q) s += part[(q * 16 * MT + t) * 33 + n];
    if (bias != nullptr) s += __bfloat162float(bias[n0 + n]);
    out[(int64_t)(t0 + t) * out_ld + n0 + n] = s;
  }
}

}  // namespace xllm

// x [T, K] with row stride x_ld, w [N, K] dense, bias [N] or null, out fp32 [T, N] with row stride out_ld.  A result does
// not depend on T: both forms add the same terms in the same order.
XLLM_API int xllm_proj_f32(void* out, int64_t out_ld, const void* x, int64_t x_ld, const void* w, const void* bias, int T, int N,
                           int K, void* stream) {
  using namespace xllm;
  if (T == 0 || N == 0) return 0;
  if (K <= 0 || K % 8 || x_ld % 8 || (((uintptr_t)x | (uintptr_t)w) & 15)) return (int)cudaErrorInvalidValue;
  const auto run = [&](auto kernel, int mt) {
    const size_t smem = (size_t)kProjWarps * 16 * mt * 33 * 4;
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    launch_pdl(kernel, dim3((T + 16 * mt - 1) / (16 * mt), (N + 31) / 32), dim3(32 * kProjWarps), smem, (cudaStream_t)stream,
               (float*)out, out_ld, (const bf16*)x, x_ld, (const bf16*)w, (const bf16*)bias, T, N, K);
    return XLLM_LAUNCH_CHECK();
  };
  return T <= 1024 ? run(proj_f32_kernel<1, 4>, 1) : run(proj_f32_kernel<2, 2>, 2);
}
