// Row kernels of decoders whose residual stream is kept in fp32, for bf16 and fp32 activations: scaled embedding,
// post-norm + residual add + pre-norm in one pass, residual sum + norm + router (or token shift) in one pass, token shift of
// whole segments, per-head query / key norm + partial rotary embedding + value mixing + paged KV append, rotary table from arbitrary frequencies, act(gate) * up,
// and a CUDA-core GEMM, dense or over row groups, for fp32 operands (and for bf16 shapes the tcgen05 kernel's TMA cannot
// address).
#include "dmoe_kernels.h"
#include "row_pack.cuh"

namespace dmoe {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const float t = warp_sum(lane < nw ? red[lane] : 0.f);
  __syncthreads();
  return t;
}

// out[t] = table[ids[t]] * scale (+ ptab[positions[t]]), fp32
template <typename T, int VEC>
__global__ void embed_f32_kernel(const int* __restrict__ ids, const T* __restrict__ table, float scale,
                                 float* __restrict__ out, int W, int vocab, const int* __restrict__ positions,
                                 const T* __restrict__ ptab, int n_pos) {
  const long long t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) id = 0;
  const T* src = table + static_cast<long long>(id) * W;
  const T* ps = ptab != nullptr ? ptab + static_cast<long long>(min(max(positions[t], 0), n_pos - 1)) * W : nullptr;
  for (int i = threadIdx.x * VEC; i < W; i += blockDim.x * VEC) {
    float x[VEC], p[VEC] = {};
    Pack<T, VEC>::load(src + i, x);
    if (ps != nullptr) Pack<T, VEC>::load(ps + i, p);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] = x[e] * scale + p[e];
    Pack<float, VEC>::store(out + t * W + i, x);
  }
}

// r = rows != NULL ? rows[i] : i;  x = resid[r] + (y != NULL ? norm(y[r]) * post : 0);  resid[r] = x where y is given and
// no row table is; h[i] = norm(x) * pre * out_scale. norm(v) = v / sqrt(mean(v^2) + eps). One CTA per output row.
constexpr int kResMax = 32;   // elements per thread: W <= 256 * 32

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
resid_norm_kernel(float* __restrict__ resid, const T* __restrict__ y, long long ld_y, const float* __restrict__ post,
                  const float* __restrict__ pre, float out_scale, float eps, const int* __restrict__ rows,
                  T* __restrict__ h, long long ld_h, int W) {
  __shared__ float red[32];
  constexpr int NV = kResMax / VEC;
  const long long i = blockIdx.x;
  const long long r = rows != nullptr ? rows[i] : i;
  const int nvec = W / VEC;
  float x[NV][VEC];
  if (y != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int v = threadIdx.x + j * blockDim.x;
      if (v < nvec) {
        Pack<T, VEC>::load(y + r * ld_y + v * VEC, x[j]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss += x[j][e] * x[j][e];
      }
    }
    const float inv = 1.f / sqrtf(cta_sum(ss, red) / static_cast<float>(W) + eps);
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int v = threadIdx.x + j * blockDim.x;
      if (v < nvec) {
        float p[VEC], s[VEC];
        Pack<float, VEC>::load(post + v * VEC, p);
        Pack<float, VEC>::load(resid + r * W + v * VEC, s);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[j][e] = s[e] + x[j][e] * inv * p[e];
        if (rows == nullptr) Pack<float, VEC>::store(resid + r * W + v * VEC, x[j]);
      }
    }
  } else {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int v = threadIdx.x + j * blockDim.x;
      if (v < nvec) Pack<float, VEC>::load(resid + r * W + v * VEC, x[j]);
    }
  }
  if (h == nullptr) return;
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    if (threadIdx.x + j * blockDim.x < nvec) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x[j][e] * x[j][e];
    }
  }
  const float inv = out_scale / sqrtf(cta_sum(ss, red) / static_cast<float>(W) + eps);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int v = threadIdx.x + j * blockDim.x;
    if (v < nvec) {
      float p[VEC];
      Pack<float, VEC>::load(pre + v * VEC, p);
#pragma unroll
      for (int e = 0; e < VEC; ++e) p[e] *= x[j][e] * inv;
      Pack<T, VEC>::store(h + i * ld_h + v * VEC, p);
    }
  }
}

// Residual sum, norm and (optionally) router of blocks whose sublayers share a norm, TPC rows per CTA of 256 threads:
//   x = resid[r] + mult (y[r] + sum_p parts[r, p]);  resid[r] = x (unless a row table picks the rows);  h = norm(x) * w
//   router: logits z = gate_w h; scores softmax(z), or sigmoid(z); the K largest (lowest index first among equals). Sigmoid
//   scores are chosen by score + correction, among the `keep` of `groups` equal runs of neighbouring experts whose two best
//   choice scores have the largest sum. Weights: scores, divided by their sum with renorm, times wscale.
//   shift: instead of h, S rows h + (before - h) mu_s per row, `before` = the slot's last row (0 at position 0), which h replaces.
//   gate: what is added is multiplied by sigmoid(gate_z + gate_bias) first; side: y is side_scale times the sum of two rows, each
//   divided by its root mean square and multiplied by its weights; bias: of the norm; conv: h and, n rows further, h + the causal
//   convolution of h with the rows in the slot's ring, which takes h.
// h_f32: h is stored as fp32.
// The rows stay in shared memory (fp32) from the sum on; with several rows per CTA the router's weights are fetched once for
// all of them.
struct SumNormArgs {
  float* resid;
  const void* y;
  long long ld_y;
  const void* parts;
  int n_parts;
  long long part_row, part_stride;
  const float* w;
  int centred;
  float eps;
  const int* rows;
  void* h;
  long long ld_h;
  int n, W;
  const void* gate_w;
  int E, K, renorm;
  int* ids;
  float* wts;
  int* counts;
  float mult;
  int h_f32;
  int sigmoid, groups, keep;
  const float* correction;
  float wscale;
  DmoeShift shift;            // n_mix = 0: none
  const float* bias;
  const void* gate_z;
  long long ld_gate;
  const float* gate_bias;
  const void* side;
  long long ld_side, side_stride;
  const float* side_w;
  float side_scale;
  DmoeConv conv;              // taps = 0: none
};
// Segment of row i of a batch of one-token segments: {row, tokens (0: padding), slot, position}
template <typename A>
__device__ __forceinline__ int4 single_segment(const A& s, long long i) {
  if (s.singles != nullptr) return static_cast<const int4*>(s.singles)[i];
  return make_int4(static_cast<int>(i), s.kv_slots[i] >= 0 ? 1 : 0, s.rows[i], s.positions[i]);
}
constexpr int kSumThreads = 256, kSumWarps = kSumThreads / 32;
constexpr int kMaxExperts = 256, kMaxTop = 32;

// add += sum over the two sides of row / root mean square (with the scale: inv) * weights, columns v * VEC ..
template <typename T, int VEC>
__device__ __forceinline__ void add_sides(const T* side, long long stride, const float* w, int W, const float (&inv)[2], int v,
                                          float* add) {
#pragma unroll
  for (int s = 0; s < 2; ++s) {
    float t[VEC], f[VEC];
    Pack<T, VEC>::load(side + s * stride + v * VEC, t);
    Pack<float, VEC>::load(w + static_cast<long long>(s) * W + v * VEC, f);
#pragma unroll
    for (int e = 0; e < VEC; ++e) add[e] += t[e] * inv[s] * f[e];
  }
}

// Row i of h (columns v * VEC .., as stored) -> its convolved row; the ring of the row's slot takes x.
template <typename T, int VEC>
__device__ __forceinline__ void convolve_single(const SumNormArgs& a, long long i, int v, const float* x) {
  const int4 seg = single_segment(a.conv, i);
  const int R = a.conv.taps, W = a.W, pos = seg.w;
  const bool live = seg.y > 0 && seg.z >= 0 && seg.z < a.conv.n_slots;
  T* ring = static_cast<T*>(a.conv.ring) + (live ? static_cast<long long>(seg.z) * R * W : 0) + v * VEC;
  float y[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) y[e] = x[e];
  for (int j = R - 1; j >= 0; --j) {
    float t[VEC], w[VEC];
    if (j > 0 && !(live && pos - j >= 0)) continue;
    if (j > 0) Pack<T, VEC>::load(ring + static_cast<long long>((pos - j) % R) * W, t);
    Pack<float, VEC>::load(a.conv.w + static_cast<long long>(R - 1 - j) * W + v * VEC, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] += w[e] * (j > 0 ? t[e] : x[e]);
  }
  if (live && R > 1) Pack<T, VEC>::store(ring + static_cast<long long>(pos % R) * W, x);
  Pack<T, VEC>::store(static_cast<T*>(a.h) + (a.n + i) * a.ld_h + v * VEC, y);
}

template <typename T, int VEC, int TPC>
__global__ void __launch_bounds__(kSumThreads) sum_norm_kernel(const SumNormArgs a) {
  constexpr int G = kSumThreads / TPC, GW = G / 32;       // threads / warps per row
  extern __shared__ __align__(16) float s_row[];          // [TPC][W]
  __shared__ float red[kSumWarps];
  __shared__ float slog[TPC][kMaxExperts];                // logits, then choice scores
  __shared__ float sscore[TPC][kMaxExperts], sgroup[TPC][kMaxExperts];      // sigmoid router: scores, sums of the groups
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int j = threadIdx.x / G, tid = threadIdx.x % G;
  const int W = a.W, nvec = W / VEC;
  const long long i = static_cast<long long>(blockIdx.x) * TPC + j;
  const bool valid = i < a.n;
  const long long r = !valid ? 0 : a.rows != nullptr ? a.rows[i] : i;
  float* row = s_row + static_cast<long long>(j) * W;
  const T* y = static_cast<const T*>(a.y);
  const T* parts = static_cast<const T*>(a.parts);
  auto group_sum = [&](float v) {       // over the threads of one row; all threads of the CTA call it
    v = warp_sum(v);
    if (GW == 1) return v;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int k = 0; k < GW; ++k) t += red[j * GW + k];
    return t;
  };

  float sinv[2] = {0.f, 0.f};           // side_scale / root mean square of the two rows
  const T* side = static_cast<const T*>(a.side) + (a.side != nullptr ? r * a.ld_side : 0);
  if (a.side != nullptr) {
#pragma unroll
    for (int s = 0; s < 2; ++s) {
      float ss = 0.f;
      if (valid)
        for (int v = tid; v < nvec; v += G) {
          float t[VEC];
          Pack<T, VEC>::load(side + s * a.side_stride + v * VEC, t);
#pragma unroll
          for (int e = 0; e < VEC; ++e) ss += t[e] * t[e];
        }
      sinv[s] = a.side_scale / sqrtf(group_sum(ss) / static_cast<float>(W) + a.eps);
    }
  }
  float sum = 0.f;
  if (valid) {
    for (int v = tid; v < nvec; v += G) {
      float x[VEC], t[VEC];
      Pack<float, VEC>::load(a.resid + r * W + v * VEC, x);
      if (a.gate_z != nullptr) {
        // the sublayer's result first, then its gate
        float add[VEC] = {};
        if (y != nullptr) Pack<T, VEC>::load(y + r * a.ld_y + v * VEC, add);
        for (int p = 0; p < a.n_parts; ++p) {
          Pack<T, VEC>::load(parts + r * a.part_row + p * a.part_stride + v * VEC, t);
#pragma unroll
          for (int e = 0; e < VEC; ++e) add[e] += t[e];
        }
        if (a.side != nullptr) add_sides<T, VEC>(side, a.side_stride, a.side_w, W, sinv, v, add);
        float z[VEC];
        Pack<T, VEC>::load(static_cast<const T*>(a.gate_z) + r * a.ld_gate + v * VEC, z);
        Pack<float, VEC>::load(a.gate_bias + v * VEC, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += a.mult * add[e] / (1.f + expf(-(z[e] + t[e])));
        if (a.rows == nullptr) Pack<float, VEC>::store(a.resid + r * W + v * VEC, x);
        Pack<float, VEC>::store(row + v * VEC, x);
#pragma unroll
        for (int e = 0; e < VEC; ++e) sum += x[e];
        continue;
      }
      if (a.side != nullptr) {
        float add[VEC] = {};
        add_sides<T, VEC>(side, a.side_stride, a.side_w, W, sinv, v, add);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += a.mult * add[e];
      }
      if (y != nullptr) {
        Pack<T, VEC>::load(y + r * a.ld_y + v * VEC, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += a.mult * t[e];
      }
      for (int p = 0; p < a.n_parts; ++p) {
        Pack<T, VEC>::load(parts + r * a.part_row + p * a.part_stride + v * VEC, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += a.mult * t[e];
      }
      if (a.rows == nullptr && (y != nullptr || a.n_parts > 0 || a.side != nullptr)) Pack<float, VEC>::store(a.resid + r * W + v * VEC, x);
      Pack<float, VEC>::store(row + v * VEC, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) sum += x[e];
    }
  }
  const float mean = a.centred ? group_sum(sum) / static_cast<float>(W) : 0.f;
  float ss = 0.f;
  if (valid)
    for (int v = tid; v < nvec; v += G)        // every thread reads back what it wrote itself
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float d = row[v * VEC + e] - mean;
        ss += d * d;
      }
  const float inv = 1.f / sqrtf(group_sum(ss) / static_cast<float>(W) + a.eps);
  if (a.shift.n_mix > 0) {
    if (!valid) return;
    const int4 seg = single_segment(a.shift, i);
    const bool live = seg.y > 0 && seg.z >= 0 && seg.z < a.shift.n_slots;
    float* last = a.shift.last + (live ? static_cast<long long>(seg.z) * W : 0);
    for (int v = tid; v < nvec; v += G) {
      float x[VEC], w[VEC], b[VEC] = {};
      Pack<float, VEC>::load(row + v * VEC, x);
      Pack<float, VEC>::load(a.w + v * VEC, w);
      if (live && seg.w > 0) Pack<float, VEC>::load(last + v * VEC, b);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] = (x[e] - mean) * inv * w[e];
      if (live) Pack<float, VEC>::store(last + v * VEC, x);
      for (int s = 0; s < a.shift.n_mix; ++s) {
        Pack<float, VEC>::load(a.shift.mu + s * W + v * VEC, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[e] = x[e] + (b[e] - x[e]) * w[e];
        Pack<T, VEC>::store(static_cast<T*>(a.h) + s * a.shift.mix_stride + i * a.ld_h + v * VEC, w);
      }
    }
    return;
  }
  if (valid)
    for (int v = tid; v < nvec; v += G) {
      float x[VEC], w[VEC];
      Pack<float, VEC>::load(row + v * VEC, x);
      Pack<float, VEC>::load(a.w + v * VEC, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] = (x[e] - mean) * inv * w[e];
      if (a.bias != nullptr) {
        Pack<float, VEC>::load(a.bias + v * VEC, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += w[e];
      }
      if (a.h_f32) {
        Pack<float, VEC>::store(static_cast<float*>(a.h) + i * a.ld_h + v * VEC, x);
        continue;
      }
      Pack<T, VEC>::store(static_cast<T*>(a.h) + i * a.ld_h + v * VEC, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] = static_cast<float>(static_cast<T>(x[e]));
      if (a.conv.taps > 0) convolve_single<T, VEC>(a, i, v, x);
      else Pack<float, VEC>::store(row + v * VEC, x);
    }
  if (a.gate_w == nullptr) return;
  __syncthreads();

  const T* gate = static_cast<const T*>(a.gate_w);
  constexpr int EB = TPC == 8 ? 4 : TPC;      // experts per pass of a warp: they share the reads of the rows
  for (int e0 = warp * EB; e0 < a.E; e0 += kSumWarps * EB) {
    float acc[EB][TPC] = {};
    for (int v = lane; v < nvec; v += 32) {
      float g[EB][VEC];
#pragma unroll
      for (int k = 0; k < EB; ++k)
        Pack<T, VEC>::load(gate + static_cast<long long>(min(e0 + k, a.E - 1)) * W + v * VEC, g[k]);
#pragma unroll
      for (int t = 0; t < TPC; ++t) {
        float x[VEC];
        Pack<float, VEC>::load(s_row + static_cast<long long>(t) * W + v * VEC, x);
#pragma unroll
        for (int k = 0; k < EB; ++k)
#pragma unroll
          for (int c = 0; c < VEC; ++c) acc[k][t] += g[k][c] * x[c];
      }
    }
#pragma unroll
    for (int k = 0; k < EB; ++k)
#pragma unroll
      for (int t = 0; t < TPC; ++t) {
        const float z = warp_sum(acc[k][t]);
        if (lane == 0 && e0 + k < a.E) slog[t][e0 + k] = z;
      }
  }
  __syncthreads();
  const long long tok = static_cast<long long>(blockIdx.x) * TPC + warp;
  if (warp >= TPC || tok >= a.n) return;
  float* lg = slog[warp];
  float* score = sscore[warp];
  float mx = -INFINITY, den = 0.f;
  if (a.sigmoid) {
    for (int e = lane; e < a.E; e += 32) {
      score[e] = 1.f / (1.f + expf(-lg[e]));
      lg[e] = score[e] + (a.correction != nullptr ? a.correction[e] : 0.f);
    }
    __syncwarp();
    if (a.keep < a.groups) {
      const int per = a.E / a.groups;
      float* sum = sgroup[warp];
      for (int g = lane; g < a.groups; g += 32) {
        float first = -INFINITY, second = -INFINITY;
        for (int e = g * per; e < (g + 1) * per; ++e) {
          const float c = lg[e];
          if (c > first) { second = first; first = c; }
          else if (c > second) second = c;
        }
        sum[g] = per > 1 ? first + second : first;
      }
      __syncwarp();
      for (int g = lane; g < a.groups; g += 32) {
        int ahead = 0;
        for (int q = 0; q < a.groups; ++q) ahead += sum[q] > sum[g] || (sum[q] == sum[g] && q < g);
        if (ahead >= a.keep)
          for (int e = g * per; e < (g + 1) * per; ++e) lg[e] = -INFINITY;
      }
      __syncwarp();
    }
  } else {
    for (int e = lane; e < a.E; e += 32) mx = fmaxf(mx, lg[e]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    for (int e = lane; e < a.E; e += 32) den += expf(lg[e] - mx);
    den = warp_sum(den);
  }
  int my_id = -1;           // lane k keeps the k-th choice
  float my_w = 0.f, total = 0.f;
  for (int k = 0; k < a.K; ++k) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < a.E; e += 32)
      if (lg[e] > best) { best = lg[e]; bi = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
    }
    float s = a.sigmoid ? (bi < a.E ? score[bi] : 0.f) : expf(best - mx) / den;
    if (bi >= a.E) {        // no finite logit left: the lowest expert not chosen yet, so that the ids stay valid
      for (bi = 0; __any_sync(0xffffffffu, my_id == bi);) ++bi;
      s = 0.f;
    }
    if (lane == k) { my_id = bi; my_w = s; }
    total += s;
    __syncwarp();
    if (lane == 0) lg[bi] = -INFINITY;
    __syncwarp();
  }
  if (lane < a.K) {
    a.ids[tok * a.K + lane] = my_id;
    a.wts[tok * a.K + lane] = (a.renorm && total > 0.f ? my_w / total : my_w) * a.wscale;
    if (a.counts != nullptr) atomicAdd(&a.counts[my_id], 1);
  }
}

// Token shift of a batch that holds longer segments: rows h (fp32) -> S mixed rows h + (before - h) mu_s, `before` = the row before
// of the same segment or, for its first row, the slot's last row. grid.x: the one-token segments, then the chunks of the longer ones
// (int4 {first row, tokens, segment, number in the segment}); grid.y: runs of kShiftRows rows of a chunk; grid.z: columns. The
// thread that reads the slot's old row writes the new one, the segment's last.
constexpr int kShiftRows = 16, kShiftThreads = 128, kMaxMix = 8;

template <typename T, int VEC>
__global__ void __launch_bounds__(kShiftThreads)
token_shift_kernel(const float* __restrict__ h, const DmoeShift a, const int4* __restrict__ multi, const int4* __restrict__ chunks,
                   T* __restrict__ out, long long ld, int W) {
  int row0, n, slot, pos0, last_row = -1;       // rows [row0, row0 + n); last_row >= 0: row0 starts its segment, which ends there
  bool first;
  if (blockIdx.x < a.n_single) {
    if (blockIdx.y > 0) return;
    const int4 seg = single_segment(a, blockIdx.x);
    if (seg.y <= 0) return;
    row0 = last_row = seg.x; n = 1; slot = seg.z; pos0 = seg.w; first = true;
  } else {
    const int4 ck = chunks[blockIdx.x - a.n_single];
    const int4 seg = multi[ck.z];
    const int skip = blockIdx.y * kShiftRows;
    if (skip >= ck.y) return;
    row0 = ck.x + skip; n = min(kShiftRows, ck.y - skip); slot = seg.z; pos0 = seg.w;
    first = row0 == seg.x;
    last_row = seg.x + seg.y - 1;
  }
  if (slot < 0 || slot >= a.n_slots) return;
  const int c = (blockIdx.z * kShiftThreads + threadIdx.x) * VEC;
  if (c >= W) return;
  float b[VEC] = {};
  float* last = a.last + static_cast<long long>(slot) * W + c;
  if (!first) Pack<float, VEC>::load(h + (row0 - 1ll) * W + c, b);
  else {
    if (pos0 > 0) Pack<float, VEC>::load(last, b);
    float x[VEC];
    Pack<float, VEC>::load(h + static_cast<long long>(last_row) * W + c, x);
    Pack<float, VEC>::store(last, x);
  }
  for (int s0 = 0; s0 < a.n_mix; s0 += 3) {          // mixing factors of three outputs at a time in registers
    float mu[3][VEC], p[VEC];
#pragma unroll
    for (int s = 0; s < 3; ++s)
      if (s0 + s < a.n_mix) Pack<float, VEC>::load(a.mu + (s0 + s) * static_cast<long long>(W) + c, mu[s]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) p[e] = b[e];
    for (int t = 0; t < n; ++t) {
      float x[VEC], y[VEC];
      Pack<float, VEC>::load(h + static_cast<long long>(row0 + t) * W + c, x);
#pragma unroll
      for (int s = 0; s < 3; ++s) {
        if (s0 + s >= a.n_mix) break;
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = x[e] + (p[e] - x[e]) * mu[s][e];
        Pack<T, VEC>::store(out + (s0 + s) * a.mix_stride + static_cast<long long>(row0 + t) * ld + c, y);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) p[e] = x[e];
    }
  }
}

// table[pos][i] = (cos, sin)(pos * freq[i]) * mscale, angles and functions in double precision
__global__ void rope_freq_table_kernel(float2* __restrict__ table, int max_pos, int half, const double* __restrict__ freq,
                                       float mscale) {
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= static_cast<long long>(max_pos) * half) return;
  double s, c;
  sincos(static_cast<double>(i / half) * freq[i % half], &s, &c);
  table[i] = make_float2(static_cast<float>(c * mscale), static_cast<float>(s * mscale));
}

// rows [q heads | k heads | v heads] (the last two only where n_kv > 0): RMS norm over each q / k head with its weight (qw !=
// NULL), rotation of the pairs (i, i + rot / 2) or, interleaved, (2i, 2i + 1), i < rot / 2, q written back in place, k and v
// appended to the paged caches ([blocks, block_size, n_kv, dk] and [.., dv]) at slots[t] (< 0: skip). v_first != NULL: what is
// appended is (1 - lambda) v + lambda v_first (head size first_head in memory). tied: rows end after the k heads, and the values
// are the first dv dimensions of every k head as it stands there, not rotated. One warp per head.
template <typename T>
__global__ void __launch_bounds__(256)
qk_norm_rope_kernel(T* __restrict__ qkv, long long ld, const int* __restrict__ positions,
                    const long long* __restrict__ slots, T* __restrict__ kcache, T* __restrict__ vcache, int n_q, int n_kv,
                    int dk, int dv, int rot, int interleaved, const float2* __restrict__ table, int max_pos,
                    const float* __restrict__ qw, const float* __restrict__ kw, float eps, const T* __restrict__ v_first,
                    long long ld_first, int first_head, float v_lambda, int tied, int v_norm) {
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int half = rot / 2;
  const int pos = min(max(positions[t], 0), max_pos - 1);
  const long long slot = slots[t];
  T* row = qkv + t * ld;
  const float2* tab = table + static_cast<long long>(pos) * half;
  for (int head = warp; head < n_q + n_kv; head += nw) {
    T* p = row + head * dk;
    const bool is_q = head < n_q;
    if (!is_q && slot < 0) continue;
    const float* w = is_q ? qw : kw;
    T* dst = is_q ? p : kcache + (slot * n_kv + (head - n_q)) * dk;
    float inv = 1.f;
    if (w != nullptr) {
      float ss = 0.f;
      for (int d = lane; d < dk; d += 32) {
        const float x = static_cast<float>(p[d]);
        ss += x * x;
      }
      inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(dk) + eps);
    }
    for (int i = lane; i < half; i += 32) {
      const int a = interleaved ? 2 * i : i, b = interleaved ? 2 * i + 1 : i + half;
      float u = static_cast<float>(p[a]), v = static_cast<float>(p[b]);
      if (w != nullptr) { u *= inv * w[a]; v *= inv * w[b]; }
      const float2 cs = tab[i];
      dst[a] = static_cast<T>(u * cs.x - v * cs.y);
      dst[b] = static_cast<T>(v * cs.x + u * cs.y);
    }
    if (w == nullptr && is_q) continue;         // the rest of the head is in place
    for (int d = rot + lane; d < dk; d += 32) {
      const float x = static_cast<float>(p[d]);
      dst[d] = static_cast<T>(w != nullptr ? x * inv * w[d] : x);
    }
  }
  if (slot >= 0) {
    const T* src = row + static_cast<long long>(tied ? n_q : n_q + n_kv) * dk;
    T* dst = vcache + slot * n_kv * dv;
    for (int head = warp; v_norm > 0 && head < n_kv; head += nw) {
      float ss = 0.f;
      for (int d = lane; d < dv; d += 32) {
        const float x = static_cast<float>(src[head * dv + d]);
        ss += x * x;
      }
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(v_norm) + eps);
      for (int d = lane; d < dv; d += 32) dst[head * dv + d] = static_cast<T>(static_cast<float>(src[head * dv + d]) * inv);
    }
    for (int i = threadIdx.x; v_norm == 0 && i < n_kv * dv; i += blockDim.x) {
      if (v_first == nullptr) { dst[i] = src[tied ? i / dv * dk + i % dv : i]; continue; }
      const int d = i % dv;
      const float first = d < first_head ? static_cast<float>(v_first[t * ld_first + i / dv * first_head + d]) : 0.f;
      dst[i] = static_cast<T>((1.f - v_lambda) * static_cast<float>(src[i]) + v_lambda * first);
    }
  }
}

// The same without norms where everything moves in 16-byte units (dk, dv and rot multiples of 8; rot / 2 too where pairs are
// half a rotation apart): the units of a row's heads are dealt out to the threads, a unit of first halves together with the unit
// of its second halves.
__global__ void __launch_bounds__(256)
rope_append_kernel(bf16* __restrict__ qkv, long long ld, const int* __restrict__ positions, const long long* __restrict__ slots,
                   bf16* __restrict__ kcache, bf16* __restrict__ vcache, int n_q, int n_kv, int dk, int dv, int rot,
                   int interleaved, const float2* __restrict__ table, int max_pos, const bf16* __restrict__ v_first,
                   long long ld_first, int first_head, float v_lambda, int tied, int v_norm, float eps) {
  const long long t = blockIdx.x;
  const int pos = min(max(positions[t], 0), max_pos - 1);
  const long long slot = slots[t];
  bf16* row = qkv + t * ld;
  const float2* tab = table + static_cast<long long>(pos) * (rot / 2);
  const int uq = n_q * dk / 8, uk = uq + (slot >= 0 ? n_kv * dk / 8 : 0);
  for (int u = threadIdx.x + (rot == 0 ? uq : 0); u < uk; u += blockDim.x) {       // without a rotation q is in place
    const int d = u * 8 % dk;
    const bool is_q = u < uq;
    if (is_q && d >= rot) continue;           // in place already
    if (!interleaved && d >= rot / 2 && d < rot) continue;      // goes with its first half
    bf16* dst = is_q ? row + u * 8 : kcache + slot * n_kv * dk + (u - uq) * 8;
    float x[8];
    Pack<bf16, 8>::load(row + u * 8, x);
    if (!interleaved && d < rot) {
      float y[8];
      Pack<bf16, 8>::load(row + u * 8 + rot / 2, y);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float2 cs = tab[d + e];
        const float p = x[e], q = y[e];
        x[e] = p * cs.x - q * cs.y;
        y[e] = q * cs.x + p * cs.y;
      }
      Pack<bf16, 8>::store(dst + rot / 2, y);
    } else if (d < rot) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 cs = tab[d / 2 + e];
        const float a = x[2 * e], b = x[2 * e + 1];
        x[2 * e] = a * cs.x - b * cs.y;
        x[2 * e + 1] = b * cs.x + a * cs.y;
      }
    }
    Pack<bf16, 8>::store(dst, x);
  }
  if (slot < 0) return;
  const bf16* src = row + static_cast<long long>(tied ? n_q : n_q + n_kv) * dk;
  bf16* dst = vcache + slot * n_kv * dv;
  if (v_norm > 0) {                               // `lanes` threads of a warp per head
    int lanes = 1;
    while (lanes < dv / 8) lanes *= 2;
    const int l = threadIdx.x & (lanes - 1);
    for (int h0 = 0; h0 < n_kv; h0 += blockDim.x / lanes) {
      const int head = h0 + threadIdx.x / lanes;
      const bool on = head < n_kv && l < dv / 8;
      float x[8] = {}, ss = 0.f;
      if (on) Pack<bf16, 8>::load(src + head * dv + l * 8, x);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
      for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = 1.f / sqrtf(ss / static_cast<float>(v_norm) + eps);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] *= inv;
      if (on) Pack<bf16, 8>::store(dst + head * dv + l * 8, x);
    }
    return;
  }
  for (int u = threadIdx.x; u < n_kv * dv / 8; u += blockDim.x) {
    float x[8];
    Pack<bf16, 8>::load(src + (tied ? u * 8 / dv * dk + u * 8 % dv : u * 8), x);
    if (v_first != nullptr) {
      const int h = u * 8 / dv, d = u * 8 % dv;
      float y[8] = {};
      if (d < first_head) Pack<bf16, 8>::load(v_first + t * ld_first + h * first_head + d, y);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = (1.f - v_lambda) * x[e] + v_lambda * y[e];
    }
    Pack<bf16, 8>::store(dst + u * 8, x);
  }
}

// out[t, i] = act(gu[t, i]) * gu[t, I + i] (act, limit, recs: see DmoeGemm)
template <typename T>
__global__ void gate_mul_kernel(const T* __restrict__ gu, long long ld, T* __restrict__ out, long long ld_out, int I, int act,
                                float limit, const int4* __restrict__ recs) {
  const long long t = blockIdx.y;
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= I) return;
  const float s = recs != nullptr ? __int_as_float(recs[t].z) : 1.f;
  const float g = static_cast<float>(gu[t * ld + i]) * s, u = static_cast<float>(gu[t * ld + I + i]) * s;
  if (act == 3) {
    const float m = fminf(g, limit);
    out[t * ld_out + i] = static_cast<T>(m / (1.f + expf(-1.702f * m)) * (fminf(fmaxf(u, -limit), limit) + 1.f));
    return;
  }
  const float v = act == 0 ? g / (1.f + expf(-g))
                           : 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
  out[t * ld_out + i] = static_cast<T>(v * u);
}

// Y[t, f] = sum_k X[t, k] W[f, k] with fp32 multiply-adds: 64 x 64 tiles, 4 x 4 outputs per thread. With offs, W is a stack of
// G matrices [F, K] and group g has rows offs[g] .. offs[g + 1] (blockIdx.y counts row tiles group after group); with recs, row
// t is scaled (not with `unit`) and stored where its record {buffer, row or < 0, weight bits, -} says. act 2: tanh of the output, 4:
// silu of its first act_cols columns.
constexpr int kSgTile = 64, kSgK = 16;

template <typename T, typename TY>
__global__ void __launch_bounds__(256)
simt_gemm_kernel(const T* __restrict__ X, long long ldx, const T* __restrict__ W, long long ldw, TY* __restrict__ Y,
                 long long ldy, int M, int F, int K, const int* __restrict__ offs, int G, const int4* __restrict__ recs,
                 void* const* __restrict__ bases, int act, int act_cols, int unit) {
  __shared__ float sx[kSgK][kSgTile + 4], sw[kSgK][kSgTile + 4];
  int t0 = blockIdx.y * kSgTile, t1 = M;
  const int f0 = blockIdx.x * kSgTile;
  if (offs != nullptr) {
    int left = blockIdx.y, g = 0;
    for (; g < G; ++g) {
      const int tiles = (offs[g + 1] - offs[g] + kSgTile - 1) / kSgTile;
      if (left < tiles) break;
      left -= tiles;
    }
    if (g == G) return;
    t0 = offs[g] + left * kSgTile;
    t1 = min(M, offs[g + 1]);
    W += static_cast<long long>(g) * F * ldw;
  }
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kSgK) {
    for (int i = threadIdx.x; i < kSgTile * kSgK; i += 256) {
      const int r = i / kSgK, k = i % kSgK;
      const bool in_k = k0 + k < K;
      sx[k][r] = in_k && t0 + r < t1 ? static_cast<float>(X[(t0 + r) * ldx + k0 + k]) : 0.f;
      sw[k][r] = in_k && f0 + r < F ? static_cast<float>(W[(f0 + r) * ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sx[k][ty * 4 + i]; b[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + ty * 4 + i;
    if (t >= t1) continue;
    TY* dst = Y + t * ldy;
    float scale = 1.f;
    if (recs != nullptr) {
      const int4 rec = recs[t];
      if (rec.y < 0) continue;
      dst = static_cast<TY*>(bases[rec.x]) + rec.y * ldy;
      scale = unit ? 1.f : __int_as_float(rec.z);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int f = f0 + tx * 4 + j;
      const float v = acc[i][j];
      if (f < F) dst[f] = static_cast<TY>(act == 2 ? tanhf(v) : act == 4 && f < act_cols ? v / (1.f + expf(-v)) : v * scale);
    }
  }
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
static int launch_resid_norm(float* resid, const void* y, long long ld_y, const float* post, const float* pre,
                             float out_scale, float eps, const int* rows, void* h, long long ld_h, int n, int W,
                             cudaStream_t stream) {
  const bool vec = W % 8 == 0 && ld_y % 8 == 0 && ld_h % 8 == 0 && aligned16(resid) && aligned16(y) && aligned16(post) &&
                   aligned16(pre) && aligned16(h);
  const int per = vec ? 8 : 1;
  int threads = ((W + per - 1) / per + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  if (W > threads * kResMax) return -10;
  if (vec)
    resid_norm_kernel<T, 8><<<n, threads, 0, stream>>>(resid, static_cast<const T*>(y), ld_y, post, pre, out_scale, eps, rows,
                                                       static_cast<T*>(h), ld_h, W);
  else
    resid_norm_kernel<T, 1><<<n, threads, 0, stream>>>(resid, static_cast<const T*>(y), ld_y, post, pre, out_scale, eps, rows,
                                                       static_cast<T*>(h), ld_h, W);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int VEC>
static int launch_sum_norm(const SumNormArgs& a, cudaStream_t stream) {
  // rows per CTA: one until there are rows for all SMs; more where a router's weights are read for every CTA
  const bool routed = a.gate_w != nullptr;
  int tpc = !routed || a.n < 160 ? 1 : a.n < 640 ? 2 : 8;
  while (tpc > 1 && static_cast<long long>(tpc) * a.W * 4 > 160 * 1024) tpc = tpc == 8 ? 2 : 1;
  const size_t smem = static_cast<size_t>(tpc) * a.W * 4;
  if (smem > 160 * 1024) return -10;
  static PerDeviceOnce configured;
  const int rc = configured.run([] {
    int e = static_cast<int>(cudaFuncSetAttribute(sum_norm_kernel<T, VEC, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    if (e == 0) e = static_cast<int>(cudaFuncSetAttribute(sum_norm_kernel<T, VEC, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    if (e == 0) e = static_cast<int>(cudaFuncSetAttribute(sum_norm_kernel<T, VEC, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    return e;
  });
  if (rc != 0) return rc;
  const unsigned grid = static_cast<unsigned>((a.n + tpc - 1) / tpc);
  if (tpc == 8) sum_norm_kernel<T, VEC, 8><<<grid, kSumThreads, smem, stream>>>(a);
  else if (tpc == 2) sum_norm_kernel<T, VEC, 2><<<grid, kSumThreads, smem, stream>>>(a);
  else sum_norm_kernel<T, VEC, 1><<<grid, kSumThreads, smem, stream>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace dmoe

using namespace dmoe;

extern "C" int dmoe_embed_f32(const int* ids, const void* table, int is_f32, float scale, float* out, int T, int W, int vocab,
                              const int* positions, const void* pos_table, int n_pos, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (W < 1 || vocab < 1 || (pos_table != nullptr && (positions == nullptr || n_pos < 1))) return -10;
  if (T == 0) return 0;
  const bool vec = W % 8 == 0 && aligned16(table) && aligned16(pos_table) && aligned16(out);
  const int threads = W >= (vec ? 2048 : 256) ? 256 : 64;
#define DMOE_EMBED(T_, VEC_)                                                                                                  \
  embed_f32_kernel<T_, VEC_><<<T, threads, 0, stream>>>(ids, static_cast<const T_*>(table), scale, out, W, vocab, positions, \
                                                        static_cast<const T_*>(pos_table), n_pos)
  if (is_f32 && vec) DMOE_EMBED(float, 8);
  else if (is_f32) DMOE_EMBED(float, 1);
  else if (vec) DMOE_EMBED(bf16, 8);
  else DMOE_EMBED(bf16, 1);
#undef DMOE_EMBED
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_resid_norm(int is_f32, float* resid, const void* y, long long ld_y, const float* post, const float* pre,
                               float out_scale, float eps, const int* rows, void* h, long long ld_h, int n, int W,
                               void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (W < 1 || resid == nullptr || (y != nullptr && post == nullptr) || (h != nullptr && pre == nullptr)) return -10;
  if (n == 0) return 0;
  return is_f32 ? launch_resid_norm<float>(resid, y, ld_y, post, pre, out_scale, eps, rows, h, ld_h, n, W, stream)
                : launch_resid_norm<bf16>(resid, y, ld_y, post, pre, out_scale, eps, rows, h, ld_h, n, W, stream);
}

extern "C" int dmoe_rope_freq_table(void* table, int max_pos, int half, const double* freq, float mscale, void* stream) {
  if (max_pos < 1 || half < 1) return -10;
  const long long n = static_cast<long long>(max_pos) * half;
  rope_freq_table_kernel<<<static_cast<unsigned>((n + 255) / 256), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<float2*>(table), max_pos, half, freq, mscale);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_sum_norm(int is_f32, float* resid, const void* y, long long ld_y, const void* parts, int n_parts,
                             long long part_row, long long part_stride, float mult, const float* w, int centred, float eps,
                             const int* rows, void* h, int h_f32, long long ld_h, int n, int W, const DmoeRouter* router,
                             const DmoeShift* shift, const DmoeSumExtra* extra, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (W < 1 || resid == nullptr || h == nullptr || w == nullptr || n_parts < 0) return -10;
  static const DmoeRouter no_router = {};
  static const DmoeShift no_shift = {};
  const DmoeRouter& r = router != nullptr ? *router : no_router;
  const DmoeShift& s = shift != nullptr ? *shift : no_shift;
  if (router != nullptr && (r.weight == nullptr || r.E < 1 || r.E > kMaxExperts || r.K < 1 || r.K > kMaxTop || r.K > r.E ||
                            r.ids == nullptr || r.wts == nullptr || h_f32 || shift != nullptr)) return -10;
  if (r.sigmoid && (r.groups < 1 || r.E % r.groups != 0 || r.keep < 1)) return -10;
  if (shift != nullptr && (rows != nullptr || s.n_single != n || s.n_mix < 1 || s.mu == nullptr || s.last == nullptr ||
                           (s.singles == nullptr && (s.positions == nullptr || s.rows == nullptr || s.kv_slots == nullptr)))) return -10;
  static const DmoeSumExtra no_extra = {};
  static const DmoeConv no_conv = {};
  const DmoeSumExtra& x = extra != nullptr ? *extra : no_extra;
  const DmoeConv& c = x.conv != nullptr ? *x.conv : no_conv;
  if ((x.gate_z != nullptr && x.gate_bias == nullptr) || (x.side != nullptr && (x.side_w == nullptr || y != nullptr))) return -10;
  if (shift != nullptr && x.bias != nullptr) return -10;
  if (x.conv != nullptr && (rows != nullptr || router != nullptr || shift != nullptr || h_f32 || c.n_single != n || c.taps < 1 ||
                            c.w == nullptr || c.ring == nullptr || c.n_slots < 1 ||
                            (c.singles == nullptr && (c.positions == nullptr || c.rows == nullptr || c.kv_slots == nullptr)))) return -10;
  if (n == 0) return 0;
  if (parts == nullptr) n_parts = 0;
  const SumNormArgs a{resid, y, ld_y, parts, n_parts, part_row, part_stride, w, centred, eps, rows, h, ld_h, n, W, r.weight, r.E,
                      r.K, r.renorm, r.ids, r.wts, r.counts, mult, h_f32, r.sigmoid, r.groups, r.keep, r.correction, r.wscale, s,
                      x.bias, x.gate_z, x.ld_gate, x.gate_bias, x.side, x.ld_side, x.side_stride, x.side_w, x.side_scale, c};
  const bool vec = W % 8 == 0 && ld_y % 8 == 0 && ld_h % 8 == 0 && part_row % 8 == 0 && part_stride % 8 == 0 && aligned16(resid) &&
                   aligned16(y) && aligned16(parts) && aligned16(w) && aligned16(h) && aligned16(r.weight) && aligned16(s.mu) &&
                   aligned16(s.last) && s.mix_stride % 8 == 0 && aligned16(x.bias) && aligned16(x.gate_z) && aligned16(x.gate_bias) &&
                   aligned16(x.side) && aligned16(x.side_w) && x.ld_gate % 8 == 0 && x.ld_side % 8 == 0 && x.side_stride % 8 == 0 &&
                   aligned16(c.w) && aligned16(c.ring);
  if (is_f32) return vec ? launch_sum_norm<float, 8>(a, stream) : launch_sum_norm<float, 1>(a, stream);
  return vec ? launch_sum_norm<bf16, 8>(a, stream) : launch_sum_norm<bf16, 1>(a, stream);
}

extern "C" int dmoe_token_shift(int is_f32, const float* h, const DmoeShift* s, const void* multi, int n_multi, const void* chunks,
                                int n_chunks, void* out, long long ld, int W, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (W < 1 || h == nullptr || out == nullptr || s->n_mix < 1 || s->n_mix > kMaxMix || s->mu == nullptr || s->last == nullptr) return -10;
  if (s->n_single < 0 || n_chunks < 0 || (n_chunks > 0 && (multi == nullptr || chunks == nullptr || n_multi < 1))) return -10;
  if (s->n_single > 0 && s->singles == nullptr && (s->positions == nullptr || s->rows == nullptr || s->kv_slots == nullptr)) return -10;
  if (s->n_single + n_chunks == 0) return 0;
  const bool vec = W % 8 == 0 && ld % 8 == 0 && s->mix_stride % 8 == 0 && aligned16(h) && aligned16(out) && aligned16(s->mu) &&
                   aligned16(s->last);
  const int per = kShiftThreads * (vec ? 8 : 1);
  const dim3 grid(s->n_single + n_chunks, n_chunks > 0 ? 64 / kShiftRows : 1, (W + per - 1) / per);
  const int4* mt = static_cast<const int4*>(multi);
  const int4* ck = static_cast<const int4*>(chunks);
#define DMOE_SHIFT(T_, VEC_) token_shift_kernel<T_, VEC_><<<grid, kShiftThreads, 0, stream>>>(h, *s, mt, ck, static_cast<T_*>(out), ld, W)
  if (is_f32 && vec) DMOE_SHIFT(float, 8);
  else if (is_f32) DMOE_SHIFT(float, 1);
  else if (vec) DMOE_SHIFT(bf16, 8);
  else DMOE_SHIFT(bf16, 1);
#undef DMOE_SHIFT
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_qk_norm_rope(int is_f32, void* qkv, long long ld, const int* positions, const long long* slots,
                                 void* kcache, void* vcache, int T, int n_q, int n_kv, int dk, int dv, int rot, int interleaved,
                                 const void* table, int max_pos, const float* qw, const float* kw, float eps,
                                 const void* v_first, long long ld_first, int first_head, float v_lambda, int tied, int v_norm,
                                 void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (n_q < 1 || n_kv < 0 || dk < 1 || rot < 0 || rot % 2 != 0 || rot > dk || (rot > 0 && table == nullptr)) return -10;
  if (n_kv > 0 && (kcache == nullptr || vcache == nullptr || (qw != nullptr && kw == nullptr))) return -10;
  if (v_first != nullptr && (first_head < 1 || tied)) return -10;
  if (tied && dv > dk) return -10;
  if (v_norm < 0 || (v_norm > 0 && (tied || v_first != nullptr || v_norm > dv))) return -10;
  if (T == 0) return 0;
  int threads = (n_q + n_kv) * 32;
  if (threads > 256) threads = 256;
  if (!is_f32 && qw == nullptr && n_kv > 0 && (v_norm == 0 || dv <= 256) && dk % 8 == 0 && dv % 8 == 0 && rot % (interleaved ? 8 : 16) == 0 &&
      ld % 8 == 0 && first_head % 8 == 0 && ld_first % 8 == 0 && aligned16(qkv) && aligned16(kcache) && aligned16(vcache) &&
      aligned16(v_first)) {
    if (rot == 0) {                              // only what is appended moves
      threads = (n_kv * (dk > dv ? dk : dv) / 8 + 31) / 32 * 32;
      if (threads > 256) threads = 256;
    }
    rope_append_kernel<<<T, threads, 0, stream>>>(
        static_cast<bf16*>(qkv), ld, positions, slots, static_cast<bf16*>(kcache), static_cast<bf16*>(vcache), n_q, n_kv, dk, dv,
        rot, interleaved, static_cast<const float2*>(table), max_pos, static_cast<const bf16*>(v_first), ld_first, first_head,
        v_lambda, tied, v_norm, eps);
    return static_cast<int>(cudaGetLastError());
  }
  if (is_f32)
    qk_norm_rope_kernel<float><<<T, threads, 0, stream>>>(
        static_cast<float*>(qkv), ld, positions, slots, static_cast<float*>(kcache), static_cast<float*>(vcache), n_q, n_kv,
        dk, dv, rot, interleaved, static_cast<const float2*>(table), max_pos, qw, kw, eps, static_cast<const float*>(v_first),
        ld_first, first_head, v_lambda, tied, v_norm);
  else
    qk_norm_rope_kernel<bf16><<<T, threads, 0, stream>>>(
        static_cast<bf16*>(qkv), ld, positions, slots, static_cast<bf16*>(kcache), static_cast<bf16*>(vcache), n_q, n_kv, dk,
        dv, rot, interleaved, static_cast<const float2*>(table), max_pos, qw, kw, eps, static_cast<const bf16*>(v_first),
        ld_first, first_head, v_lambda, tied, v_norm);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_gate_mul(int is_f32, int act, const void* gu, long long ld, void* out, long long ld_out, int T, int I,
                             float limit, const void* recs, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (I < 1 || (act != 0 && act != 1 && act != 3)) return -10;
  for (int t0 = 0; t0 < T; t0 += 65535) {      // grid.y limit
    const int n = T - t0 < 65535 ? T - t0 : 65535;
    const dim3 grid((I + 255) / 256, n);
    const int4* rc = recs != nullptr ? static_cast<const int4*>(recs) + t0 : nullptr;
    if (is_f32)
      gate_mul_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const float*>(gu) + t0 * ld, ld,
                                                       static_cast<float*>(out) + t0 * ld_out, ld_out, I, act, limit, rc);
    else
      gate_mul_kernel<bf16><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(gu) + t0 * ld, ld,
                                                      static_cast<bf16*>(out) + t0 * ld_out, ld_out, I, act, limit, rc);
  }
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_simt_linear(int x_f32, int y_f32, const void* X, long long ldx, const void* W, long long ldw, void* Y,
                                long long ldy, int T, int F, int K, int act, int act_cols, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (F < 1 || K < 1 || (x_f32 && !y_f32)) return -10;
  if (T == 0) return 0;
  const long long ty = (T + kSgTile - 1) / kSgTile;
  if (ty > 65535) return -10;
  const dim3 grid((F + kSgTile - 1) / kSgTile, static_cast<unsigned>(ty));
  if (x_f32)
    simt_gemm_kernel<float, float><<<grid, 256, 0, stream>>>(static_cast<const float*>(X), ldx, static_cast<const float*>(W),
                                                             ldw, static_cast<float*>(Y), ldy, T, F, K, nullptr, 0, nullptr, nullptr, act, act_cols, 0);
  else if (y_f32)
    simt_gemm_kernel<bf16, float><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(X), ldx, static_cast<const bf16*>(W), ldw,
                                                            static_cast<float*>(Y), ldy, T, F, K, nullptr, 0, nullptr, nullptr, act, act_cols, 0);
  else
    simt_gemm_kernel<bf16, bf16><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(X), ldx, static_cast<const bf16*>(W), ldw,
                                                           static_cast<bf16*>(Y), ldy, T, F, K, nullptr, 0, nullptr, nullptr, act, act_cols, 0);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_simt_grouped(int is_f32, int y_f32, const void* X, long long ldx, const void* W, const int* offs, int G, void* Y,
                                 long long ldy, const void* recs, const void* bases, int unit_weights, int T, int F, int K,
                                 void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (F < 1 || K < 1 || G < 1 || offs == nullptr || (recs == nullptr && Y == nullptr) || (recs != nullptr && bases == nullptr)) return -10;
  if (T == 0) return 0;
  const long long ty = (T + kSgTile - 1) / kSgTile + G;      // every group may end in a partial tile
  if (ty > 65535) return -10;
  const dim3 grid((F + kSgTile - 1) / kSgTile, static_cast<unsigned>(ty));
  const int4* r = static_cast<const int4*>(recs);
  void* const* b = static_cast<void* const*>(bases);
  if (is_f32)
    simt_gemm_kernel<float, float><<<grid, 256, 0, stream>>>(static_cast<const float*>(X), ldx, static_cast<const float*>(W), K,
                                                             static_cast<float*>(Y), ldy, T, F, K, offs, G, r, b, 0, 0, unit_weights);
  else if (y_f32)
    simt_gemm_kernel<bf16, float><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(X), ldx, static_cast<const bf16*>(W), K,
                                                            static_cast<float*>(Y), ldy, T, F, K, offs, G, r, b, 0, 0, unit_weights);
  else
    simt_gemm_kernel<bf16, bf16><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(X), ldx, static_cast<const bf16*>(W), K,
                                                           static_cast<bf16*>(Y), ldy, T, F, K, offs, G, r, b, 0, 0, unit_weights);
  return static_cast<int>(cudaGetLastError());
}
