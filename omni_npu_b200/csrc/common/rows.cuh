// Rows of bf16 or fp32 read and written as floats, eight (16 or 32 bytes) or four elements at a time.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

namespace b200 {

template <typename T>
struct Row8;
template <>
struct Row8<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const void* base, long long vec, float (&v)[8]) {
    const uint4 u = reinterpret_cast<const uint4*>(base)[vec];
    const uint32_t r[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = __uint_as_float(r[i] << 16);
      v[2 * i + 1] = __uint_as_float(r[i] & 0xffff0000u);
    }
  }
  static __device__ __forceinline__ void store(void* base, long long vec, const float (&v)[8]) {
    uint4 u;
    uint32_t* r = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 p = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
      r[i] = *reinterpret_cast<const uint32_t*>(&p);
    }
    reinterpret_cast<uint4*>(base)[vec] = u;
  }
};
template <>
struct Row8<float> {
  static __device__ __forceinline__ void load(const void* base, long long vec, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4*>(base)[2 * vec];
    const float4 b = reinterpret_cast<const float4*>(base)[2 * vec + 1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
  static __device__ __forceinline__ void store(void* base, long long vec, const float (&v)[8]) {
    reinterpret_cast<float4*>(base)[2 * vec] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(base)[2 * vec + 1] = make_float4(v[4], v[5], v[6], v[7]);
  }
};

// The same four elements (8 or 16 bytes) at a time.
template <typename T>
struct Row4;
template <>
struct Row4<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const void* base, long long vec, float (&v)[4]) {
    const uint2 u = reinterpret_cast<const uint2*>(base)[vec];
    v[0] = __uint_as_float(u.x << 16);
    v[1] = __uint_as_float(u.x & 0xffff0000u);
    v[2] = __uint_as_float(u.y << 16);
    v[3] = __uint_as_float(u.y & 0xffff0000u);
  }
  static __device__ __forceinline__ void store(void* base, long long vec, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    reinterpret_cast<uint2*>(base)[vec] =
        make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
};
template <>
struct Row4<float> {
  static __device__ __forceinline__ void load(const void* base, long long vec, float (&v)[4]) {
    const float4 a = reinterpret_cast<const float4*>(base)[vec];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  }
  static __device__ __forceinline__ void store(void* base, long long vec, const float (&v)[4]) {
    reinterpret_cast<float4*>(base)[vec] = make_float4(v[0], v[1], v[2], v[3]);
  }
};

__device__ __forceinline__ float as_float(float x) { return x; }
__device__ __forceinline__ float as_float(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T>
__device__ __forceinline__ T from_float(float x);
template <>
__device__ __forceinline__ float from_float<float>(float x) { return x; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float x) { return __float2bfloat16(x); }

}  // namespace b200
