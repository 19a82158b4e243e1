// V (4 or 1) neighbouring values loaded as float32, and stored as float32 or rounded to the array's type.
#pragma once
#include "common.cuh"

namespace pbe {

template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&a)[V]) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    a[0] = v.x; a[1] = v.y; a[2] = v.z; a[3] = v.w;
  } else {
    a[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void load_v(const __nv_bfloat16* p, float (&a)[V]) {
  if constexpr (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    a[0] = lo.x; a[1] = lo.y; a[2] = hi.x; a[3] = hi.y;
  } else {
    a[0] = __bfloat162float(*p);
  }
}
template <int V>
__device__ __forceinline__ void put_v(float* p, const float (&a)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a[0], a[1], a[2], a[3]);
  else *p = a[0];
}
template <int V>
__device__ __forceinline__ void put_v(__nv_bfloat16* p, const float (&a)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a[0], a[1]), hi = __floats2bfloat162_rn(a[2], a[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
  } else {
    *p = __float2bfloat16_rn(a[0]);
  }
}

}  // namespace pbe
