// Groups of VW adjacent values of a row (VW 4: one 16- or 8-byte access, VW 1: any alignment).
#pragma once
#include "pk_common.cuh"

namespace pk {

template <int VW>
__device__ __forceinline__ void load_f32(const float* p, float (&v)[VW]) {
  if (VW == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1 % VW] = x.y; v[2 % VW] = x.z; v[3 % VW] = x.w;
  } else {
    v[0] = *p;
  }
}
template <int VW>
__device__ __forceinline__ void store(float* p, const float (&v)[VW]) {
  if (VW == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % VW], v[2 % VW], v[3 % VW]);
  else *p = v[0];
}
template <int VW>
__device__ __forceinline__ void store(bf16* p, const float (&v)[VW]) {
  if (VW == 4) {
    const bf162 a = __floats2bfloat162_rn(v[0], v[1 % VW]), b = __floats2bfloat162_rn(v[2 % VW], v[3 % VW]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16(v[0]);
  }
}

template <int VW>
__device__ __forceinline__ void load_any(const void* p, size_t at, bool f32, float (&v)[VW]) {
  if (f32) {
    load_f32<VW>((const float*)p + at, v);
  } else if (VW == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>((const bf16*)p + at);
    v[0] = __uint_as_float(u.x << 16); v[1 % VW] = __uint_as_float(u.x & 0xffff0000u);
    v[2 % VW] = __uint_as_float(u.y << 16); v[3 % VW] = __uint_as_float(u.y & 0xffff0000u);
  } else {
    v[0] = __bfloat162float(((const bf16*)p)[at]);
  }
}

}  // namespace pk
