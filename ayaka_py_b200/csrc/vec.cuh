// One or four numbers at a time between 32-bit registers and memory; four: 16-byte loads, 8- or 16-byte stores.
#pragma once

#include "common.cuh"

__device__ __forceinline__ void store_n(float* dst, const float (&v)[1]) { *dst = v[0]; }
__device__ __forceinline__ void store_n(__nv_bfloat16* dst, const float (&v)[1]) { *dst = __float2bfloat16_rn(v[0]); }
__device__ __forceinline__ void store_n(float* dst, const float (&v)[4]) { *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store_n(__nv_bfloat16* dst, const float (&v)[4]) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  uint2 packed;
  packed.x = *reinterpret_cast<uint32_t*>(&lo);
  packed.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(dst) = packed;
}
__device__ __forceinline__ void load_n(const float* src, float (&v)[1]) { v[0] = *src; }
__device__ __forceinline__ void load_n(const float* src, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(src);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
