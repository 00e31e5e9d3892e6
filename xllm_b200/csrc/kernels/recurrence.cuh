// Token-by-token recurrences over a matrix state S [dk, dv] held in registers, for prompt chunks.
//
// A warp owns eight state columns: lane = 8 * column group + row group, a lane holds two neighbouring columns of the
// rows 4 (r + 8 j) .. + 3 (j < J), so that the eight row groups read a token's key-sized vectors from shared memory as
// one contiguous 128-byte line per j and the four column groups by broadcast.  Columns never meet: a token needs two
// sums over the eight row groups (three shuffles each) and no barrier; warps meet once per tile of tokens, when the next
// tile's vectors are staged.  All arithmetic is fp32, two rows per instruction (fma.rn.f32x2).
#pragma once
#include "common.cuh"

namespace xllm {

typedef unsigned long long f2;      // two packed floats

__device__ __forceinline__ f2 pack_f2(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack_f2(f2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f2 fma_f2(f2 a, f2 b, f2 c) {
  f2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f2 mul_f2(f2 a, f2 b) {
  f2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f2 add_f2(f2 a, f2 b) {
  f2 d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

constexpr int kRecTile = 16;        // tokens staged together
constexpr int kRecCols = 8;         // state columns of a warp

template <int J>
struct StateColumns {
  f2 s[2][2 * J];                   // [column][pair of rows]

  // S: the head's state [dk, dv_pad] at this lane's first column
  __device__ __forceinline__ void load(const float* S, int dk, int dv_pad, int row_group, bool live) {
#pragma unroll
    for (int j = 0; j < J; ++j)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int r = 4 * (row_group + 8 * j) + e;
        float2 a = make_float2(0.f, 0.f), b = a;
        if (live && r < dk) a = *reinterpret_cast<const float2*>(S + (int64_t)r * dv_pad);
        if (live && r + 1 < dk) b = *reinterpret_cast<const float2*>(S + (int64_t)(r + 1) * dv_pad);
        s[0][2 * j + e / 2] = pack_f2(a.x, b.x);
        s[1][2 * j + e / 2] = pack_f2(a.y, b.y);
      }
  }
  __device__ __forceinline__ void store(float* S, int dk, int dv_pad, int row_group) const {
#pragma unroll
    for (int j = 0; j < J; ++j)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int r = 4 * (row_group + 8 * j) + e;
        const float2 a = unpack_f2(s[0][2 * j + e / 2]), b = unpack_f2(s[1][2 * j + e / 2]);
        if (r < dk) *reinterpret_cast<float2*>(S + (int64_t)r * dv_pad) = make_float2(a.x, b.x);
        if (r + 1 < dk) *reinterpret_cast<float2*>(S + (int64_t)(r + 1) * dv_pad) = make_float2(a.y, b.y);
      }
  }
};

// this lane's rows of a key-sized vector in shared memory (zero behind dk)
template <int J>
__device__ __forceinline__ void load_rows(const float* v, int row_group, f2* out) {
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(v + 4 * (row_group + 8 * j));
    out[2 * j] = u.x;
    out[2 * j + 1] = u.y;
  }
}

// sum over the eight row groups, in every lane
__device__ __forceinline__ float sum_row_groups(float v) {
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  return v;
}
// the same for two columns at once: an even lane gets the first column's sum, an odd lane the second's
__device__ __forceinline__ float sum_row_groups_2(float a, float b) {
  const bool odd = threadIdx.x & 1;
  const float give = odd ? a : b, keep = odd ? b : a;
  float v = keep + __shfl_xor_sync(0xffffffffu, give, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  return v;
}

}  // namespace xllm
