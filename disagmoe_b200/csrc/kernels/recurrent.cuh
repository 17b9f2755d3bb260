// Shared pieces of the recurrence kernels: gates and decays in fp32, the convolution step, small loads.
#pragma once
#include "dmoe_kernels.h"
#include "sm100.cuh"

namespace dmoe {

constexpr int kMaxTaps = 8;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// log of the decay of one key channel: kind 0: log sigmoid(z) * scale, kind 1: -scale * softplus(z)
__device__ __forceinline__ float log_decay(int kind, float z, float scale) {
  return kind == 0 ? -softplus(-z) * scale : -scale * softplus(z);
}
__device__ __forceinline__ float gate_value(int kind, float g) { return (kind == 0 ? g : 1.f) / (1.f + expf(-g)); }

// Segment i of a decode step: row i alone.
__device__ __forceinline__ int4 row_segment(const DmoeRecur& a, int i) {
  return make_int4(i, a.kv_slots[i] >= 0 ? 1 : 0, a.rows[i], a.positions[i]);
}

template <int VEC>
__device__ __forceinline__ void load_vec(const float* p, float* f) {
  if (VEC == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x;
    if (VEC == 4) { f[VEC - 3] = v.y; f[VEC - 2] = v.z; f[VEC - 1] = v.w; }
  } else {
    f[0] = p[0];
  }
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* p, const float* f) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[VEC - 3], f[VEC - 2], f[VEC - 1]);
  else p[0] = f[0];
}

// Convolution + silu of one channel of a one-token segment at position pos, from the raw projection `src` and the ring of
// earlier inputs (ring[slot][p % taps][channel]); the one writing thread of a channel stores the new input. Slot
// pos % taps is not among the taps - 1 positions that are read, so readers in other CTAs do not race with it.
template <typename T>
__device__ __forceinline__ float conv_step(const DmoeRecur& a, long long row, int pos, int slot, int channel,
                                           const void* src, long long ld, int src_col, bool writes) {
  const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim, R = a.taps;
  T* ring = static_cast<T*>(a.ring) + static_cast<long long>(slot) * R * C + channel;
  const float* w = a.conv_w + static_cast<long long>(channel) * R;
  const T x = static_cast<const T*>(src)[row * ld + src_col];
  float acc = 0.f;
  for (int j = R - 1; j >= 1; --j)
    if (pos - j >= 0) acc += w[R - 1 - j] * static_cast<float>(ring[static_cast<long long>((pos - j) % R) * C]);
  acc += w[R - 1] * static_cast<float>(x);
  if (writes && R > 1) ring[static_cast<long long>(pos % R) * C] = x;
  return static_cast<float>(static_cast<T>(silu(acc)));
}

}  // namespace dmoe
