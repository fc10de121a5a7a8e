// Loads and stores of one or four elements of float32 or bf16 as float32.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common.cuh"

namespace ferrl {

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 o;
  o.x = *reinterpret_cast<uint32_t*>(&a);
  o.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = o;
}
// V elements per access: 4 where width, strides and addresses allow it, else 1
template <int V> struct Vec { float v[V]; };
template <int V, typename T> __device__ __forceinline__ Vec<V> ld(const T* p) {
  Vec<V> r;
  if constexpr (V == 4) {
    const float4 f = load4(p);
    r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
  } else {
    r.v[0] = to_f(*p);
  }
  return r;
}
template <int V, typename T> __device__ __forceinline__ void st(T* p, const Vec<V>& r) {
  if constexpr (V == 4) store4(p, make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
  else *p = from_f<T>(r.v[0]);
}

}  // namespace ferrl
