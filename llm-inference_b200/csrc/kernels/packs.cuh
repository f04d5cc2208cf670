// Rows read and written four numbers at a time as 32-bit values (16-byte accesses of float, 8-byte ones of bfloat16), or
// one at a time where a row's length or alignment does not allow that: kernels are written once over `Pack<W>`.
#pragma once

#include "common.cuh"

template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <>
__device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <>
__device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v);
template <>
__device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <>
__device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<uint32_t*>(&lo);
  raw.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = raw;
}

__device__ __forceinline__ float fma_each(float a, float b, float c) { return fmaf(a, b, c); }
__device__ __forceinline__ float4 fma_each(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
__device__ __forceinline__ float4 fma_each(float4 a, float b, float4 c) {
  return make_float4(fmaf(a.x, b, c.x), fmaf(a.y, b, c.y), fmaf(a.z, b, c.z), fmaf(a.w, b, c.w));
}
__device__ __forceinline__ float scale_each(float a, float s) { return a * s; }
__device__ __forceinline__ float4 scale_each(float4 a, float s) { return make_float4(a.x * s, a.y * s, a.z * s, a.w * s); }
__device__ __forceinline__ float mul_each(float a, float b) { return a * b; }
__device__ __forceinline__ float4 mul_each(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float add_each(float a, float b) { return a + b; }
__device__ __forceinline__ float4 add_each(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float sub_each(float a, float b) { return a - b; }
__device__ __forceinline__ float4 sub_each(float4 a, float4 b) { return make_float4(a.x - b.x, a.y - b.y, a.z - b.z, a.w - b.w); }
__device__ __forceinline__ float square_sum(float a, float acc) { return fmaf(a, a, acc); }
__device__ __forceinline__ float square_sum(float4 a, float acc) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, fmaf(a.w, a.w, acc)))); }

// W numbers per access: 4 (rows whose length is a multiple of four, aligned) or 1.
template <int W>
struct Pack;
template <>
struct Pack<4> {
  using type = float4;
  template <typename T>
  static __device__ __forceinline__ float4 load(const T* p) { return load4<T>(p); }
  template <typename T>
  static __device__ __forceinline__ void store(T* p, float4 v) { store4<T>(p, v); }
};
template <>
struct Pack<1> {
  using type = float;
  template <typename T>
  static __device__ __forceinline__ float load(const T* p) { return to_f32<T>(*p); }
  template <typename T>
  static __device__ __forceinline__ void store(T* p, float v) { *p = from_f32<T>(v); }
};

inline bool packs_of_four(int count) { return count % 4 == 0; }
template <typename... Rest>
bool packs_of_four(int count, const void* p, Rest... rest) {  // every pointer on a 16-byte boundary, rows of whole packs
  return reinterpret_cast<uintptr_t>(p) % 16 == 0 && packs_of_four(count, rest...);
}
