// Causal convolutions over time per channel, and Griffin's real-gated diagonal recurrence (De et al., "Griffin: Mixing Gated
// Linear Recurrences with Local Attention for Efficient Language Models"):
//
//   log a = decay sigmoid(r),   S <- a S + sqrt(1 - a^2) sigmoid(i) u,   out = S gelu(y)        per channel, S in fp32
//
// A step's rows fall into segments of one sequence (tables as in recurrent.cu). One-token segments take one launch of elementwise
// work; longer ones are scanned: a CTA owns some channels of a segment and walks it a few hundred tokens at a time, every thread
// a run of eight tokens of one channel. A run is a map S -> A S + B; the maps of a pass are composed in shared memory, then every
// thread goes through its run again from registers. Gates, decays and states are fp32.
#include "dmoe_kernels.h"
#include "recurrent.cuh"
#include "row_pack.cuh"

namespace dmoe {

constexpr int kConvRows = 16, kConvThreads = 128;

// {row, tokens (0: padding), slot, position} of one-token segment i
template <typename A>
__device__ __forceinline__ int4 one_token(const A& a, long long i) {
  if (a.singles != nullptr) return static_cast<const int4*>(a.singles)[i];
  return make_int4(static_cast<int>(i), a.kv_slots[i] >= 0 ? 1 : 0, a.rows[i], a.positions[i]);
}

// grid.x: the one-token segments, then the chunks of the longer ones; grid.y: runs of kConvRows rows of a chunk; grid.z: columns.
// Only the thread of a segment's first rows reads the ring, and it stores the segment's last inputs there afterwards.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kConvThreads)
seq_conv_kernel(const T* __restrict__ x, long long ldx, const DmoeConv a, const int4* __restrict__ multi,
                const int4* __restrict__ chunks, T* __restrict__ out, long long ldo, long long block_stride, int C) {
  constexpr int HIST = TAPS - 1;
  int row0, n, seg_row, seg_n, slot, pos0;        // rows [row0, row0 + n) of the segment that starts at seg_row, position pos0
  if (blockIdx.x < a.n_single) {
    if (blockIdx.y > 0) return;
    const int4 s = one_token(a, blockIdx.x);
    if (s.y <= 0) return;
    row0 = seg_row = s.x; n = seg_n = 1; slot = s.z; pos0 = s.w;
  } else {
    const int4 ck = chunks[blockIdx.x - a.n_single];
    const int4 s = multi[ck.z];
    const int skip = blockIdx.y * kConvRows;
    if (skip >= ck.y) return;
    row0 = ck.x + skip; n = min(kConvRows, ck.y - skip);
    seg_row = s.x; seg_n = s.y; slot = s.z; pos0 = s.w;
  }
  if (slot < 0 || slot >= a.n_slots) return;
  const int c = (blockIdx.z * kConvThreads + threadIdx.x) * VEC, R = a.taps;
  if (c >= C) return;
  T* ring = static_cast<T*>(a.ring) + static_cast<long long>(slot) * R * C + c;
  const int pos = pos0 + row0 - seg_row;          // position of row0
  float w[TAPS][VEC], hist[HIST > 0 ? HIST : 1][VEC], bias[VEC] = {}, add[VEC] = {};      // hist[j - 1]: the input j tokens back
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) w[j][e] = 0.f;
    if (j < R) Pack<float, VEC>::load(a.w + static_cast<long long>(R - 1 - j) * C + c, w[j]);
  }
  if (a.in_bias != nullptr) Pack<float, VEC>::load(a.in_bias + c, bias);
  if (a.out_bias != nullptr) Pack<float, VEC>::load(a.out_bias + c, add);
#pragma unroll
  for (int j = 1; j <= HIST; ++j) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) hist[j - 1][e] = 0.f;
    if (j < R && pos - j >= 0) {
      if (row0 - j >= seg_row) Pack<T, VEC>::load(x + (row0 - j) * ldx + c, hist[j - 1]);
      else Pack<T, VEC>::load(ring + static_cast<long long>((pos - j) % R) * C, hist[j - 1]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) hist[j - 1][e] += bias[e];
    }
  }
  if (row0 == seg_row) {
    for (int j = 0; j < R - 1 && j < seg_n; ++j) {
      float v[VEC];
      Pack<T, VEC>::load(x + static_cast<long long>(seg_row + seg_n - 1 - j) * ldx + c, v);
      Pack<T, VEC>::store(ring + static_cast<long long>((pos0 + seg_n - 1 - j) % R) * C, v);
    }
  }
  const int per = C / a.blocks;
  T* dst = out + (c / per) * block_stride + c % per;
#pragma unroll 4
  for (int t = 0; t < n; ++t) {
    float v[VEC], acc[VEC];
    Pack<T, VEC>::load(x + static_cast<long long>(row0 + t) * ldx + c, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      v[e] += bias[e];
      acc[e] = a.residual ? v[e] + add[e] : add[e];
#pragma unroll
      for (int j = HIST; j >= 1; --j) acc[e] += w[j][e] * hist[j - 1][e];
      acc[e] += w[0][e] * v[e];
#pragma unroll
      for (int j = HIST; j >= 2; --j) hist[j - 1][e] = hist[j - 2][e];
      if (HIST > 0) hist[0][e] = v[e];
    }
    Pack<T, VEC>::store(dst + static_cast<long long>(row0 + t) * ldo, acc);
  }
}

// ---- the recurrence ----------------------------------------------------------------------------------------------------
// x sigmoid(z); FAST: with the approximate exponential and division (fp32 to a few ulp)
template <bool FAST>
__device__ __forceinline__ float times_sigmoid(float x, float z) {
  return FAST ? __fdividef(x, 1.f + __expf(-z)) : x / (1.f + expf(-z));
}
// tanh form of gelu: z sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3))
template <bool FAST>
__device__ __forceinline__ float gelu_gate(float z) {
  return times_sigmoid<FAST>(z, 1.5957691216057308f * (z + 0.044715f * z * z * z));
}
// exp(x) - 1 for x <= 0: the Taylor series near zero (relative error below 2e-8 there), the exponential elsewhere
__device__ __forceinline__ float expm1_below(float x) {
  float p = 1.f / 5040.f;
  p = p * x + 1.f / 720.f;
  p = p * x + 1.f / 120.f;
  p = p * x + 1.f / 24.f;
  p = p * x + 1.f / 6.f;
  p = p * x + 0.5f;
  p = p * x + 1.f;
  return x > -0.35f ? p * x : __expf(x) - 1.f;
}
// a token's step: S <- a S + b. 1 - a^2 = -(a - 1) (a + 1) from a - 1 = expm1(log a), exact where a is near one
template <bool FAST>
__device__ __forceinline__ void unit_step(float r, float i, float u, float decay, float& a, float& b) {
  const float x = times_sigmoid<FAST>(decay, r), e = FAST ? expm1_below(x) : expm1f(x);
  a = 1.f + e;
  const float w = -e * (2.f + e);
  b = (FAST ? w * rsqrtf(fmaxf(w, 1e-37f)) : sqrtf(w)) * times_sigmoid<FAST>(u, i);
}

constexpr int kUnitThreads = 256;

template <typename T, int VEC>
__global__ void __launch_bounds__(kUnitThreads) unit_step_kernel(const DmoeUnit d) {
  const int4 s = one_token(d, blockIdx.x);
  if (s.y <= 0 || s.z < 0 || s.z >= d.n_slots) return;
  const int c = (blockIdx.y * kUnitThreads + threadIdx.x) * VEC, per = d.width / d.blocks;
  if (c >= d.width) return;
  const int blk = c / per, o = c % per;
  const long long at = blk * d.block_rows + s.x;
  const float* g = d.gates + at * 2 * d.padded + o;
  float* sp = d.state + static_cast<long long>(s.z) * d.width + c;
  float u[VEC], r[VEC], i[VEC], rb[VEC], ib[VEC], y[VEC], yb[VEC], dec[VEC], S[VEC] = {};
  load_any<VEC>(static_cast<const T*>(d.u) + at * d.padded + o, u);
  load_any<VEC>(g, r);
  load_any<VEC>(g + d.padded, i);
  load_any<VEC>(static_cast<const T*>(d.y) + s.x * d.ldy + c, y);
  if (s.w > 0) load_any<VEC>(sp, S);
  load_any<VEC>(d.gate_bias + 2 * blk * d.padded + o, rb);
  load_any<VEC>(d.gate_bias + (2 * blk + 1) * d.padded + o, ib);
  load_any<VEC>(d.y_bias + c, yb);
  load_any<VEC>(d.decay + c, dec);
#pragma unroll
  for (int e = 0; e < VEC; ++e) {
    float a, b;
    unit_step<sizeof(T) == 2>(r[e] + rb[e], i[e] + ib[e], u[e], dec[e], a, b);
    S[e] = a * S[e] + b;
    y[e] = S[e] * gelu_gate<sizeof(T) == 2>(y[e] + yb[e]);
  }
  store_any<VEC>(sp, S);
  store_any<VEC>(static_cast<T*>(d.out) + s.x * d.ldo + c, y);
}

constexpr int kScanThreads = 512, kRun = 8;

// CH channels per CTA; 32 / CH runs per warp
template <typename T, int CH>
__global__ void __launch_bounds__(kScanThreads) unit_scan_kernel(const DmoeUnit d) {
  constexpr int RUNS = kScanThreads / CH, PASS = RUNS * kRun;
  __shared__ float s_a[2][RUNS][CH], s_b[2][RUNS][CH], s_carry[2][CH];
  const int4 seg = static_cast<const int4*>(d.multi)[blockIdx.x];
  if (seg.y <= 0 || seg.z < 0 || seg.z >= d.n_slots) return;
  const int ch = threadIdx.x % CH, run = threadIdx.x / CH, per = d.width / d.blocks;
  const int c = blockIdx.y * CH + ch, cc = min(c, d.width - 1);
  const bool on = c < d.width;
  const int blk = cc / per, o = cc % per;
  // this run's rows, one pass further each time
  const long long row = seg.x + run * kRun;
  const T* up = static_cast<const T*>(d.u) + (blk * d.block_rows + row) * d.padded + o;
  const float* gp = d.gates + (blk * d.block_rows + row) * 2 * d.padded + o;
  const T* yp = static_cast<const T*>(d.y) + row * d.ldy + cc;
  T* op = static_cast<T*>(d.out) + row * d.ldo + cc;
  const float rb = d.gate_bias[2 * blk * d.padded + o], ib = d.gate_bias[(2 * blk + 1) * d.padded + o];
  const float yb = d.y_bias[cc], dec = d.decay[cc];
  float* sp = d.state + static_cast<long long>(seg.z) * d.width + cc;
  if (run == 0) s_carry[0][ch] = seg.w > 0 ? *sp : 0.f;

  float u[kRun], r[kRun], i[kRun], y[kRun];
  const int p = d.padded, ldy = static_cast<int>(d.ldy), ldo = static_cast<int>(d.ldo);
  auto fetch = [&](int left) {                       // left: tokens of the segment from the run's first on
    if (left >= kRun) {
#pragma unroll
      for (int k = 0; k < kRun; ++k) {
        u[k] = static_cast<float>(up[k * p]);
        r[k] = gp[2 * k * p];
        i[k] = gp[2 * k * p + p];
        y[k] = static_cast<float>(yp[k * ldy]);
      }
    } else {
#pragma unroll
      for (int k = 0; k < kRun; ++k) {
        const bool in = k < left;
        u[k] = in ? static_cast<float>(up[k * p]) : 0.f;
        r[k] = in ? gp[2 * k * p] : 0.f;
        i[k] = in ? gp[2 * k * p + p] : 0.f;
        y[k] = in ? static_cast<float>(yp[k * ldy]) : 0.f;
      }
    }
    up += static_cast<long long>(PASS) * p;
    gp += 2ll * PASS * p;
    yp += PASS * d.ldy;
  };
  fetch(seg.y - run * kRun);
  int buf = 0;
  for (int t0 = 0; t0 < seg.y; t0 += PASS, buf ^= 1) {
    const int left = seg.y - t0 - run * kRun;      // tokens of the segment from this run's first on
    float a[kRun], b[kRun], g[kRun], A = 1.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < kRun; ++k) {
      unit_step<sizeof(T) == 2>(r[k] + rb, i[k] + ib, u[k], dec, a[k], b[k]);
      if (k >= left) {
        a[k] = 1.f;
        b[k] = 0.f;
      }
      g[k] = gelu_gate<sizeof(T) == 2>(y[k] + yb);
      A *= a[k];
      B = a[k] * B + b[k];
    }
    s_a[buf][run][ch] = A;
    s_b[buf][run][ch] = B;
    if (t0 + PASS < seg.y) fetch(left - PASS);
    __syncthreads();
    float S = s_carry[buf][ch];
#pragma unroll 8
    for (int j = 0; j < run; ++j) S = s_a[buf][j][ch] * S + s_b[buf][j][ch];
#pragma unroll
    for (int k = 0; k < kRun; ++k) {
      S = a[k] * S + b[k];
      if (on && k < left) op[k * ldo] = static_cast<T>(S * g[k]);
    }
    op += PASS * d.ldo;
    // tokens past the end leave S alone: the last run ends with the state of the segment's last token
    if (run == RUNS - 1) {
      s_carry[buf ^ 1][ch] = S;
      if (on && t0 + PASS >= seg.y) *sp = S;
    }
  }
}

template <typename T>
static int run_unit(const DmoeUnit& d, cudaStream_t stream) {
  if (d.n_single > 0) {
    const int per = d.width / d.blocks;
    const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = per % 4 == 0 && d.ldy % 4 == 0 && d.ldo % 4 == 0 && al(d.u) && al(d.gates) && al(d.y) && al(d.out) && al(d.state) &&
                     al(d.gate_bias) && al(d.y_bias) && al(d.decay);
    const int cols = kUnitThreads * (vec ? 4 : 1);
    const dim3 grid(d.n_single, (d.width + cols - 1) / cols);
    if (vec) unit_step_kernel<T, 4><<<grid, kUnitThreads, 0, stream>>>(d);
    else unit_step_kernel<T, 1><<<grid, kUnitThreads, 0, stream>>>(d);
  }
  if (d.n_multi > 0) {
    // fewer channels per CTA where the wide ones would leave SMs idle
    if (static_cast<long long>(d.n_multi) * ((d.width + 31) / 32) >= device_num_sms())
      unit_scan_kernel<T, 32><<<dim3(d.n_multi, (d.width + 31) / 32), kScanThreads, 0, stream>>>(d);
    else
      unit_scan_kernel<T, 16><<<dim3(d.n_multi, (d.width + 15) / 16), kScanThreads, 0, stream>>>(d);
  }
  return static_cast<int>(cudaGetLastError());
}

}  // namespace dmoe

using namespace dmoe;

extern "C" int dmoe_seq_conv(int is_f32, const void* x, long long ldx, const DmoeConv* a, const void* multi, int n_multi,
                             const void* chunks, int n_chunks, void* out, long long ldo, long long block_stride, int C, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (C < 1 || x == nullptr || out == nullptr || a->w == nullptr || a->ring == nullptr || a->n_slots < 1) return -10;
  if (a->taps < 1 || a->taps > kMaxTaps || a->blocks < 1 || C % a->blocks != 0 || a->n_single < 0 || n_chunks < 0) return -11;
  if (n_chunks > 0 && (multi == nullptr || chunks == nullptr || n_multi < 1)) return -12;
  if (a->n_single > 0 && a->singles == nullptr && (a->positions == nullptr || a->rows == nullptr || a->kv_slots == nullptr)) return -12;
  if (a->n_single + n_chunks == 0) return 0;
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = C % 8 == 0 && C / a->blocks % 8 == 0 && ldx % 8 == 0 && ldo % 8 == 0 && block_stride % 8 == 0 && al(x) && al(out) &&
                   al(a->w) && al(a->ring) && al(a->in_bias) && al(a->out_bias);
  const int per = kConvThreads * (vec ? 8 : 1);
  const dim3 grid(a->n_single + n_chunks, n_chunks > 0 ? 64 / kConvRows : 1, (C + per - 1) / per);
  const int4* mt = static_cast<const int4*>(multi);
  const int4* ck = static_cast<const int4*>(chunks);
#define DMOE_CONV(T_, VEC_)                                                                                                   \
  do {                                                                                                                       \
    const T_* xp = static_cast<const T_*>(x);                                                                                \
    T_* op = static_cast<T_*>(out);                                                                                          \
    if (a->taps <= 4) seq_conv_kernel<T_, VEC_, 4><<<grid, kConvThreads, 0, stream>>>(xp, ldx, *a, mt, ck, op, ldo, block_stride, C); \
    else seq_conv_kernel<T_, VEC_, kMaxTaps><<<grid, kConvThreads, 0, stream>>>(xp, ldx, *a, mt, ck, op, ldo, block_stride, C); \
  } while (0)
  if (is_f32 && vec) DMOE_CONV(float, 8);
  else if (is_f32) DMOE_CONV(float, 1);
  else if (vec) DMOE_CONV(bf16, 8);
  else DMOE_CONV(bf16, 1);
#undef DMOE_CONV
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_unit_recurrence(int is_f32, const DmoeUnit* d, void* stream) {
  if (d->width < 1 || d->blocks < 1 || d->width % d->blocks != 0 || d->padded < d->width / d->blocks || d->n_slots < 1) return -10;
  if (d->u == nullptr || d->gates == nullptr || d->gate_bias == nullptr || d->decay == nullptr || d->y == nullptr ||
      d->y_bias == nullptr || d->state == nullptr || d->out == nullptr) return -10;
  if (d->n_single > 0 && d->singles == nullptr && (d->positions == nullptr || d->rows == nullptr || d->kv_slots == nullptr)) return -11;
  if (d->n_multi > 0 && d->multi == nullptr) return -11;
  return is_f32 ? run_unit<float>(*d, static_cast<cudaStream_t>(stream)) : run_unit<bf16>(*d, static_cast<cudaStream_t>(stream));
}
