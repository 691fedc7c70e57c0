// Device-side readers of a projection slice (proj_src.h) and conversions between storage types and fp32.
#pragma once
#include "common.cuh"
#include "proj_src.h"

namespace nkb {
__device__ __forceinline__ float proj_load(const NkbProj& s, long long row, int col) {
  if (s.bf16) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(s.ptr)[row * s.ld + col]);
  const float* p = reinterpret_cast<const float*>(s.ptr) + row * s.ld + col;
  float a = p[0];
#pragma unroll 4
  for (int i = 1; i < s.splits; ++i) a += p[i * s.split_stride];
  return a;
}
// four consecutive columns; the host has checked that they are aligned (proj_vec4_ok)
__device__ __forceinline__ float4 proj_load4(const NkbProj& s, long long row, int col) {
  if (s.bf16) {
    const uint2 r = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(s.ptr) + row * s.ld + col);
    const float2 a = unpack_bf16x2(r.x), b = unpack_bf16x2(r.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  const float* p = reinterpret_cast<const float*>(s.ptr) + row * s.ld + col;
  float4 v = *reinterpret_cast<const float4*>(p);
#pragma unroll 4
  for (int i = 1; i < s.splits; ++i) {
    const float4 w = *reinterpret_cast<const float4*>(p + i * s.split_stride);
    v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
  }
  return v;
}
static inline bool proj_vec4_ok(const NkbProj& s) {
  const uintptr_t a = reinterpret_cast<uintptr_t>(s.ptr);
  return (a & (s.bf16 ? 7 : 15)) == 0 && (s.ld & 3) == 0 && (s.split_stride & 3) == 0;
}
// the reciprocal is the approximate one (two units in the last place): an IEEE division costs more than the exponential
__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.f, 1.f + expf(-z)); }

template <typename T>
__device__ __forceinline__ T cast_out(float v);
template <>
__device__ __forceinline__ float cast_out<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 cast_out<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
template <typename T>
__device__ __forceinline__ float cast_in(T v);
template <>
__device__ __forceinline__ float cast_in<float>(float v) { return v; }
template <>
__device__ __forceinline__ float cast_in<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
}  // namespace nkb
