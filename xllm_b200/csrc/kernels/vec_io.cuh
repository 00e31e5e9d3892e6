// Vector loads and stores of V elements of bf16 or fp32 as fp32 registers, for kernels that are
// templates over the activation type.  V = 8 and 4 need pointers aligned to V elements (16 bytes at
// most); V = 1 takes any pointer.
#pragma once
#include "common.cuh"

namespace xllm {

template <int V>
__device__ __forceinline__ void load_f32(const bf16* p, float* f) {
  if constexpr (V == 8) {
    unpack8(*reinterpret_cast<const bf16x8*>(p), f);
  } else if constexpr (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&u.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int V>
__device__ __forceinline__ void load_f32(const float* p, float* f) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(p + i);
      f[i] = a.x; f[i + 1] = a.y; f[i + 2] = a.z; f[i + 3] = a.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = p[i];
  }
}
template <int V>
__device__ __forceinline__ void store_f32(bf16* p, const float* f) {
  if constexpr (V == 8) {
    *reinterpret_cast<bf16x8*>(p) = pack8(f);
  } else if constexpr (V == 4) {
    uint2 u;
    *reinterpret_cast<bf162*>(&u.x) = __floats2bfloat162_rn(f[0], f[1]);
    *reinterpret_cast<bf162*>(&u.y) = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16(f[i]);
  }
}
template <int V>
__device__ __forceinline__ void store_f32(float* p, const float* f) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = f[i];
  }
}

// Sigmoid and silu of values whose results leave as T: hardware exponential and division (2^-21 relative) in front of a
// rounding to bf16, the accurate ones for fp32.
template <typename T>
__device__ __forceinline__ float sigmoid_as(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-z));
  else return 1.f / (1.f + expf(-z));
}
template <typename T>
__device__ __forceinline__ float silu_as(float z) { return z * sigmoid_as<T>(z); }

__device__ __forceinline__ float to_f32(bf16 x) { return __bfloat162float(x); }
__device__ __forceinline__ float to_f32(float x) { return x; }
template <typename T>
__device__ __forceinline__ T from_f32(float x);
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float x) { return __float2bfloat16(x); }
template <>
__device__ __forceinline__ float from_f32<float>(float x) { return x; }

}  // namespace xllm
