// Rows of bf16 or fp32 values as floats, one or eight neighbours per access.
#pragma once
#include "sm100.cuh"

namespace dmoe {

typedef __nv_bfloat16 bf16;

template <typename T, int VEC>
struct Pack;   // VEC elements of T <-> floats, one aligned access where VEC > 1
template <typename T>
struct Pack<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float* f) { f[0] = static_cast<float>(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float* f) { p[0] = static_cast<T>(f[0]); }
};
template <>
struct Pack<float, 8> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
  }
};
template <>
struct Pack<bf16, 8> {
  static __device__ __forceinline__ void load(const bf16* p, float* f) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 t = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
      f[2 * i] = t.x;
      f[2 * i + 1] = t.y;
    }
  }
  static __device__ __forceinline__ void store(bf16* p, const float* f) {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 t = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
      w[i] = *reinterpret_cast<const uint32_t*>(&t);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
};

}  // namespace dmoe
