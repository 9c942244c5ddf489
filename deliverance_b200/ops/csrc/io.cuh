// Loads and stores of activations that are bf16 or fp32, as fp32 values.
#pragma once
#include "common.cuh"

namespace dlv {

__device__ __forceinline__ float io_ld(const __nv_bfloat16* p) { return bf2f(*p); }
__device__ __forceinline__ float io_ld(const float* p) { return *p; }
__device__ __forceinline__ void io_st(__nv_bfloat16* p, float v) { *p = f2bf(v); }
__device__ __forceinline__ void io_st(float* p, float v) { *p = v; }
template <typename TIO>
__device__ __forceinline__ void io_ld4(const TIO* p, float* v) {
  if constexpr (sizeof(TIO) == 2) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf162(u.x), b = unpack_bf162(u.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  } else {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  }
}
template <typename TIO>
__device__ __forceinline__ void io_st4(TIO* p, const float* v) {
  if constexpr (sizeof(TIO) == 2) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf162(v[0], v[1]), pack_bf162(v[2], v[3]));
  else *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <typename TIO>
__device__ __forceinline__ void io_ld8(const TIO* p, float* v) {
  if constexpr (sizeof(TIO) == 2) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = unpack_bf162(w[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  } else {
    io_ld4(p, v);
    io_ld4(p + 4, v + 4);
  }
}
template <typename TIO>
__device__ __forceinline__ void io_st8(TIO* p, const float* v) {
  if constexpr (sizeof(TIO) == 2)
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf162(v[0], v[1]), pack_bf162(v[2], v[3]), pack_bf162(v[4], v[5]), pack_bf162(v[6], v[7]));
  else {
    io_st4(p, v);
    io_st4(p + 4, v + 4);
  }
}

}  // namespace dlv
