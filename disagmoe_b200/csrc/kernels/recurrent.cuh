// Shared pieces of the recurrence kernels: gates and decays in fp32, the convolution step, small loads.
#pragma once
#include "dmoe_kernels.h"
#include "sm100.cuh"

namespace dmoe {

constexpr int kMaxTaps = 8;
enum { kPlain = 0, kDelta = 1, kBonus = 2, kMemory = 3 };      // MODE of the kernels: how a token writes and where it reads, see recurrent.cu

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
// log(1 + e) for 0 <= e <= 1 as 2 atanh(e / (2 + e)): the odd series in s <= 1/3, to full fp32 accuracy also for tiny e
__device__ __forceinline__ float log1p_unit(float e) {
  const float s = __fdividef(e, 2.f + e), q = s * s;
  float p = 1.f / 15.f;
  p = p * q + 1.f / 13.f;
  p = p * q + 1.f / 11.f;
  p = p * q + 1.f / 9.f;
  p = p * q + 1.f / 7.f;
  p = p * q + 1.f / 5.f;
  p = p * q + 1.f / 3.f;
  return 2.f * (s + s * q * p);
}
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1p_unit(expf(-fabsf(x))); }
// log of the decay of one key channel: kind 0: log sigmoid(z) * scale, kind 1: -scale * softplus(z), kind 2: -exp(z), kind 3: scale
__device__ __forceinline__ float log_decay(int kind, float z, float scale) {
  if (kind == 2) return -expf(z);
  if (kind == 3) return scale;
  return kind == 0 ? -softplus(-z) * scale : -scale * softplus(z);
}
__device__ __forceinline__ float decay_scale(const DmoeRecur& a, int h) {
  return a.decay_kind == 0 ? a.inv_tau : a.decay_kind == 1 ? expf(a.a_log[h]) : a.decay_kind == 3 ? a.head_decay[h] : 1.f;
}
// Matrix memory: logs of the input and the forget gate of a token
__device__ __forceinline__ void memory_logs(const DmoeRecur& a, long long row, int h, float& i, float& f) {
  const float* z = a.gates + row * a.ldgates;
  i = a.gate_cap * tanhf((z[h] + a.gate_bias[h]) / a.gate_cap);
  f = -softplus(-a.gate_cap * tanhf((z[a.heads + h] + a.gate_bias[a.heads + h]) / a.gate_cap));
}
// the running maximum in the slot is kept at the parity of its position: what one CTA writes no other one of the step reads
__device__ __forceinline__ float* max_state(const DmoeRecur& a, int slot, int pos, int h) {
  return a.max_state + (static_cast<long long>(slot) * 2 + (pos & 1)) * a.heads + h;
}
// factor of a read-out: 1 / (max(|n . q|, exp(-m)) + 1e-6)
__device__ __forceinline__ float memory_scale(float nq, float m) { return 1.f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f); }
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

// VEC consecutive values of either type as floats (one access; VEC is 1, 2 or 4)
template <int VEC>
__device__ __forceinline__ void load_any(const float* p, float* f) {
  if (VEC == 4) load_vec<VEC>(p, f);
  else
    for (int i = 0; i < VEC; ++i) f[i] = p[i];
}
template <int VEC>
__device__ __forceinline__ void load_any(const __nv_bfloat16* p, float* f) {
  if (VEC == 1) {
    f[0] = __bfloat162float(p[0]);
    return;
  }
  uint32_t r[2];
  if (VEC == 4) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    r[0] = v.x;
    r[1] = v.y;
  } else {
    r[0] = r[1] = *reinterpret_cast<const uint32_t*>(p);
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r[i / 2]));
    f[i] = i % 2 ? v.y : v.x;
  }
}
template <int VEC>
__device__ __forceinline__ void store_any(float* p, const float* f) {
  if (VEC == 4) store_vec<VEC>(p, f);
  else
    for (int i = 0; i < VEC; ++i) p[i] = f[i];
}
template <int VEC>
__device__ __forceinline__ void store_any(__nv_bfloat16* p, const float* f) {
  if (VEC == 1) {
    p[0] = __float2bfloat16(f[0]);
    return;
  }
  uint32_t r[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(f[VEC == 4 ? 2 * i : 0], f[VEC == 4 ? 2 * i + 1 : VEC - 1]);
    r[i] = *reinterpret_cast<const uint32_t*>(&v);
  }
  if (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(r[0], r[1]);
  else *reinterpret_cast<uint32_t*>(p) = r[0];
}

// Convolution + silu of one channel of a one-token segment at position pos, from the raw projection and the ring of earlier
// inputs (ring[slot][p % taps][channel]). load() requests everything, finish() combines it and, in the one writing thread
// of a channel, stores the new input. Slot pos % taps is not among the taps - 1 positions that are read, so readers in
// other CTAs do not race with it.
template <typename T>
struct ConvInputs {
  T x[kMaxTaps];
  float w[kMaxTaps];
  __device__ __forceinline__ static T* ring_of(const DmoeRecur& a, int slot, int channel) {
    const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
    return static_cast<T*>(a.ring) + static_cast<long long>(slot) * a.taps * C + channel;
  }
  __device__ __forceinline__ void load(const DmoeRecur& a, long long row, int pos, int slot, int channel, const void* src,
                                       long long ld, int src_col) {
    const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim, R = a.taps;
    const T* ring = ring_of(a, slot, channel);
    const float* wp = a.conv_w + static_cast<long long>(channel) * R + R - 1;
    x[0] = static_cast<const T*>(src)[row * ld + src_col];
    w[0] = wp[0];
#pragma unroll
    for (int j = 1; j < kMaxTaps; ++j) {
      const bool on = j < R && pos - j >= 0;
      x[j] = on ? ring[static_cast<long long>((pos - j) % R) * C] : static_cast<T>(0.f);
      w[j] = on ? wp[-j] : 0.f;
    }
  }
  __device__ __forceinline__ float finish(const DmoeRecur& a, int pos, int slot, int channel, bool writes) {
    float acc = 0.f;
#pragma unroll
    for (int j = kMaxTaps - 1; j >= 0; --j) acc += w[j] * static_cast<float>(x[j]);
    const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
    if (writes && a.taps > 1) ring_of(a, slot, channel)[static_cast<long long>(pos % a.taps) * C] = x[0];
    return static_cast<float>(static_cast<T>(silu(acc)));
  }
};

}  // namespace dmoe
