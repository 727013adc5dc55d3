// One element or four neighbouring ones of a row, loaded and stored together.
#pragma once
#include "common.cuh"

template <int V> struct Vec { float f[V]; };
template <int V> __device__ __forceinline__ Vec<V> ldv(const float* p) {
  Vec<V> r;
  if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    r.f[0] = a.x; r.f[1] = a.y; r.f[2] = a.z; r.f[3] = a.w;
  } else r.f[0] = *p;
  return r;
}
template <int V> __device__ __forceinline__ void stv(void* p, int dtype, size_t i, const Vec<V>& v) {
  if constexpr (V == 4) {
    if (dtype == RUAI_F32) *reinterpret_cast<float4*>((float*)p + i) = make_float4(v.f[0], v.f[1], v.f[2], v.f[3]);
    else {
      __nv_bfloat162 a = __floats2bfloat162_rn(v.f[0], v.f[1]), b = __floats2bfloat162_rn(v.f[2], v.f[3]);
      *reinterpret_cast<uint2*>((__nv_bfloat16*)p + i) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
    }
  } else store_from_f32(p, dtype, i, v.f[0]);
}
