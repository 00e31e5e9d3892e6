// Tensor-core fragment helpers shared by the paged attention kernels.
#pragma once
#include "common.cuh"

namespace xllm {

__device__ __forceinline__ void cp_async16(uint32_t smem_addr, const void* gptr, bool valid) {
  const int sz = valid ? 16 : 0;  // src-size 0 => zero fill, nothing is read
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_addr), "l"(gptr), "r"(sz));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;\n" ::"n"(N));
}

__device__ __forceinline__ void ldmatrix_x4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3,
                                            uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t& r0, uint32_t& r1, uint32_t& r2,
                                                  uint32_t& r3, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}

// D(16x8,f32) += A(16x16,bf16,row) * B(16x8,bf16,col)
__device__ __forceinline__ void mma_bf16_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
      "{%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// D(16x8,f32) = A(16x16,bf16,row) * B(16x8,bf16,col)
__device__ __forceinline__ void mma_bf16_16816_first(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
      "{%10,%10,%10,%10};\n"
      : "=f"(c[0]), "=f"(c[1]), "=f"(c[2]), "=f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1), "f"(0.f));
}

__device__ __forceinline__ uint32_t pack_bf162(float lo, float hi) {
  bf162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// Two fp32 values as two bf16 pairs whose sum keeps about 16 bits of their significands.
__device__ __forceinline__ void split_pack(float a, float b, uint32_t& hi, uint32_t& lo) {
  const bf162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const bf162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 unpack2(uint32_t u) { return __bfloat1622float2(*reinterpret_cast<const bf162*>(&u)); }

// Scores bounded by a soft cap, in the log2 domain: cap * log2(e) * tanh(s * scale / cap) = out - 2 out / (1 + 2^(s * in))
// with in = 2 log2(e) scale / cap and out = cap log2(e).  The quotient leaves an error of a few 1e-7 of the cap.
// Scores of at most two fifths of the cap need neither: tanh(x) = x P(x^2) for |x| <= 0.4, P of degree three by the exchange
// algorithm of Remez (relative error 1e-7), and a tile of such scores is worth a vote.
struct SoftCap {
  float in, out;             // out 0: no cap
  float k[4], small;         // |s| <= small: s (k0 + k1 s^2 + k2 s^4 + k3 s^6)
};
inline SoftCap make_soft_cap(float scale, float cap) {
  const float log2e = 1.4426950408889634f;
  SoftCap c = {};
  if (!(cap > 0.f)) return c;
  const double unit = (double)scale / cap, size = unit < 0 ? -unit : unit;
  const double poly[4] = {0.9999999019, -0.3333136246, 0.1327097676, -0.04755360363};
  double f = (double)cap * log2e * unit;
  for (int i = 0; i < 4; ++i, f *= unit * unit) c.k[i] = (float)(poly[i] * f);
  c.in = (float)(2. * log2e * unit);
  c.out = cap * log2e;
  // the last coefficient must neither fade away nor overflow
  c.small = size > 1e-4 && size < 1e3 && cap < 1e4f ? (float)(0.4 / size) : -1.f;
  return c;
}
// capped score + plus
__device__ __forceinline__ float soft_cap_small(float s, const SoftCap& c, float plus = 0.f) {
  const float t = s * s;
  float p = fmaf(t, c.k[3], c.k[2]);
  p = fmaf(t, p, c.k[1]);
  p = fmaf(t, p, c.k[0]);
  return fmaf(s, p, plus);
}
__device__ __forceinline__ float soft_cap(float s, const SoftCap& c) {
  return c.out - __fdividef(2.f * c.out, 1.f + exp2f(s * c.in));
}

// Byte offset of 16-byte chunk `c` of row `r` in a tile whose rows hold CH chunks; the XOR
// swizzle makes 8 consecutive rows of one chunk column hit 8 different bank groups.
template <int CH>
__device__ __forceinline__ uint32_t swz(int r, int c) {
  return (uint32_t)((r * CH + (c ^ (r & 7))) << 4);
}

}  // namespace xllm
