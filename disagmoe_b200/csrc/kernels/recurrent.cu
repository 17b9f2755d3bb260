// Linear recurrences with a matrix-valued state per head, S [dim, vdim] in fp32, a decay per head and key channel and
// one of two writes per token (the plain one with two places of the read-out):
//
//   plain   S <- diag(a) S + k v^T                                 (gated linear attention)
//   delta   S <- diag(a) S;  S <- S + k (beta (v - S^T k))^T       (gated delta rule)
//   o = S^T q, read after the write
//   bonus   o = (S + diag(u) k v^T)^T q, then the plain write      (RWKV-style time mixing)
//   memory  the plain write with k scaled and one decay per head and token, both relative to a running maximum m of the logs of
//           the gates; o = S^T q / (max(|n.q|, e^-m) + 1e-6) with n <- a n + k            (matrix memory of xLSTM)
//
// Plain writes also come with one constant decay per head (lightning attention).
//
// States live in slots: slot = block-table row of the sequence, so a sequence's state is found with the same index as
// its KV pages, and a sequence whose first token is in the batch (position 0) starts from zero whatever the slot held.
//
// Work is described by tables that the host builds once per step:
//   segs    int4 {first row, tokens, slot, position of the first token}; a segment = consecutive rows of one sequence
//   chunks  int4 {first row, tokens <= 64, segment, chunk number in the segment}
// Segments of one token (decoding) take stream_step_kernel or step_kernel, which do everything from the raw projections to
// the gated, normalised output in one launch. Longer ones are convolved by conv_chunk_kernel and then run either through the chunked
// tensor-core kernels of recurrent_chunk.cu or, token by token in fp32 arithmetic, through step_kernel.
#include "dmoe_kernels.h"
#include "recurrent.cuh"

namespace dmoe {

constexpr int kStepThreads = 256;
constexpr int kStepRows = 16;        // state rows a thread holds in registers

// Matrix memory: decay factor, factor of k and running maximum of a token, from the arrays of dmoe_memory_gates or, for a token on
// its own, from its gates and the slot's maximum.
struct TokenGates {
  float keep, put, top;
};
__device__ __forceinline__ TokenGates token_gates(const DmoeRecur& a, long long row, int pos, int slot, int h) {
  TokenGates g;
  if (a.keep != nullptr) {
    const long long at = h * a.ldsteps + row;
    g.keep = expf(a.keep[at]);
    g.put = a.put[at];
    g.top = a.run_max[at];
    return g;
  }
  float i, f;
  memory_logs(a, row, h, i, f);
  if (pos > 0) f += *max_state(a, slot, pos - 1, h);
  g.top = fmaxf(f, i);
  g.keep = expf(f - g.top);
  g.put = expf(i - g.top);
  return g;
}

// Decay factor, q and k of the token's key channels and its values -> shared memory (convolved and activated with CONV). Matrix
// memory: with them the normaliser, which moves on in its slot (the CTA of the first value columns has it).
template <typename T, int MODE, bool CONV>
__device__ __forceinline__ void token_inputs(const DmoeRecur& a, long long row, int pos, int slot, int h, int hk, int v0, int nv,
                                             float scale, const TokenGates& tg, float4* s_gqk, float* s_v) {
  const int D = a.dim, V = a.vdim, group = a.heads / a.kv_heads;
  for (int i = threadIdx.x; i < D + nv; i += blockDim.x) {
    if (i < D) {
      const float z = MODE != kMemory && a.z != nullptr ? a.z[row * a.ldz + h * D + i] + a.z_bias[h * D + i] : 0.f;
      float q, k;
      if (CONV) {
        ConvInputs<T> xq, xk;
        xq.load(a, row, pos, slot, hk * D + i, a.q, a.ldq, hk * D + i);
        xk.load(a, row, pos, slot, (a.kv_heads + hk) * D + i, a.k, a.ldk, hk * D + i);
        const bool writes = h % group == 0 && v0 == 0;
        q = xq.finish(a, pos, slot, hk * D + i, writes);
        k = xk.finish(a, pos, slot, (a.kv_heads + hk) * D + i, writes);
      } else {
        q = static_cast<float>(static_cast<const T*>(a.q)[row * a.ldq + hk * D + i]);
        k = static_cast<float>(static_cast<const T*>(a.k)[row * a.ldk + hk * D + i]);
      }
      if (MODE == kMemory) {
        float n = 0.f;
        if (v0 == 0) {
          float* np = a.norm_state + (static_cast<long long>(slot) * a.heads + h) * D + i;
          if (pos > 0) n = *np;
          *np = tg.keep * n + tg.put * k;
        }
        s_gqk[i] = make_float4(tg.keep, q, k, n);
        continue;
      }
      s_gqk[i] = make_float4(expf(log_decay(a.decay_kind, z, scale)), q, k, MODE == kBonus ? a.bonus[h * D + i] : 0.f);
    } else {
      const int c = h * V + v0 + i - D;
      if (CONV) {
        ConvInputs<T> xv;
        xv.load(a, row, pos, slot, 2 * a.kv_heads * D + c, a.v, a.ldv, c);
        s_v[i - D] = xv.finish(a, pos, slot, 2 * a.kv_heads * D + c, true);
      } else {
        s_v[i - D] = static_cast<float>(static_cast<const T*>(a.v)[row * a.ldv + c]);
      }
    }
  }
}

// Factors that turn the raw rows into q (scaled, unit) and k (unit), and the weight of the token's own write in its read-out:
// q.k of the raw rows, with the bonus q.(u k); every warp on its own. Matrix memory: the factor of the read-out.
struct RowFactors {
  float fq, fk, qk, scale;
};
template <int MODE>
__device__ __forceinline__ RowFactors row_factors(const DmoeRecur& a, const float4* s_gqk, const TokenGates& tg) {
  float qq = 0.f, kk = 0.f, qk = 0.f, nq = 0.f;
  for (int d = threadIdx.x & 31; d < a.dim; d += 32) {
    const float4 x = s_gqk[d];
    qq += x.y * x.y;
    kk += x.z * x.z;
    qk += MODE == kBonus ? x.y * (x.z * x.w) : x.y * x.z;
    if (MODE == kMemory) nq += x.y * x.w;
  }
  RowFactors f;
  f.qk = warp_sum(qk);
  f.fq = a.qscale;
  f.fk = 1.f;
  f.scale = 1.f;
  if (MODE == kMemory) {
    f.fk = tg.put;
    f.scale = memory_scale((tg.keep * warp_sum(nq) + tg.put * f.qk) * f.fq, tg.top);
  }
  if (MODE == kDelta) {
    f.fq *= 1.f / sqrtf(warp_sum(qq) + 1e-6f);
    f.fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
  }
  return f;
}

// One CTA: one segment, one head, `vt` value columns. Threads form a grid of (vt / VEC) column groups x rpp row groups;
// a thread keeps rows rg, rg + rpp, ... of its VEC columns in registers for the whole segment. Per token the read-outs
// of the decayed (with a bonus: undecayed) state at k and at q are reduced together, and o = (a S)^T q + (k.q) u gives the
// read-out after the write without a second pass.
template <typename T, int MODE, bool CONV, int VEC>
__global__ void __launch_bounds__(kStepThreads, 2)
step_kernel(const DmoeRecur a, int vt) {
  constexpr bool DELTA = MODE == kDelta;
  extern __shared__ __align__(16) float s_mem[];
  const int tid = threadIdx.x, lane = tid & 31;
  const int4 seg = a.segs != nullptr ? static_cast<const int4*>(a.segs)[blockIdx.x] : row_segment(a, blockIdx.x);
  const int row0 = seg.x, ntok = seg.y, slot = seg.z, pos0 = seg.w;
  if (ntok <= 0 || slot < 0 || slot >= a.n_slots) return;
  const int h = blockIdx.y, D = a.dim, V = a.vdim;
  const int group = a.heads / a.kv_heads, hk = DELTA ? h / group : h;
  const int v0 = blockIdx.z * vt, nv = min(vt, V - v0);
  const int vq = vt / VEC, rpp = kStepThreads / vq;
  const int cg = tid % vq, rg = tid / vq;
  const bool mine = rg < rpp && cg * VEC < nv;
  float4* s_gqk = reinterpret_cast<float4*>(s_mem);    // [D] decay factor, q, k of the token
  float* s_v = s_mem + 4 * D;          // [vt]
  float* s_u = s_v + vt;               // [vt]
  float* s_o = s_u + vt;               // [vt]
  float* s_red = s_o + vt;             // [DELTA ? 2 : 1][rpp][vt]
  float* sp = a.state + ((static_cast<long long>(slot) * a.heads + h) * D) * V + v0 + cg * VEC;

  float S[kStepRows][VEC];
#pragma unroll
  for (int i = 0; i < kStepRows; ++i) {
    const int d = rg + i * rpp;
#pragma unroll
    for (int e = 0; e < VEC; ++e) S[i][e] = 0.f;
    if (mine && d < D && pos0 > 0) load_vec<VEC>(sp + static_cast<long long>(d) * V, S[i]);
  }
  const float dscale = decay_scale(a, h);
  const float* norm_w = a.norm_w + h * a.norm_ld;

  for (int t = 0; t < ntok; ++t) {
    const long long row = row0 + t;
    const int pos = pos0 + t;
    // what the end of the step needs, requested before anything waits
    const bool fused = a.raw == nullptr;
    const int oc = min(tid, nv - 1);
    float beta = 0.f, gate = 0.f, weight = 0.f;
    if (DELTA) beta = static_cast<float>(static_cast<const T*>(a.beta)[row * a.ldb + h]);
    if (fused) {
      gate = static_cast<float>(static_cast<const T*>(a.gate)[row * a.ldg + h * V + oc]);
      weight = norm_w[oc];
    }
    TokenGates tg = {};
    if (MODE == kMemory) {
      tg = token_gates(a, row, pos, slot, h);
      if (a.keep == nullptr && v0 == 0 && tid == 0) *max_state(a, slot, pos, h) = tg.top;
    }
    token_inputs<T, MODE, CONV>(a, row, pos, slot, h, hk, v0, nv, dscale, tg, s_gqk, s_v);
    __syncthreads();
    const RowFactors f = row_factors<MODE>(a, s_gqk, tg);
    if (MODE == kMemory && !fused && v0 == 0 && tid == 0) a.scale[row * a.heads + h] = f.scale;
    const float fq = f.fq, fk = f.fk, qk = f.qk;
    if (DELTA) beta = 1.f / (1.f + expf(-beta));
    float rq[VEC], rk[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) rq[e] = rk[e] = 0.f;
    if (mine) {
#pragma unroll
      for (int i = 0; i < kStepRows; ++i) {
        const int d = rg + i * rpp;
        if (d < D) {
          const float4 x = s_gqk[d];
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            if (MODE == kBonus) rq[e] += S[i][e] * x.y;
            S[i][e] *= x.x;
            if (MODE != kBonus) rq[e] += S[i][e] * x.y;
            if (DELTA) rk[e] += S[i][e] * x.z;
          }
        }
      }
      store_vec<VEC>(s_red + rg * vt + cg * VEC, rq);
      if (DELTA) store_vec<VEC>(s_red + (rpp + rg) * vt + cg * VEC, rk);
    }
    __syncthreads();
    for (int c = tid; c < nv; c += kStepThreads) {
      float oq = 0.f, ok = 0.f;
#pragma unroll 4
      for (int r = 0; r < rpp; ++r) {
        oq += s_red[r * vt + c];
        if (DELTA) ok += s_red[(rpp + r) * vt + c];
      }
      float u = s_v[c];
      if (DELTA) u = beta * (u - ok * fk);
      s_u[c] = u * fk;
      const float o = oq * fq + qk * fq * fk * u;
      if (fused) s_o[c] = o * f.scale;
      else a.raw[row * a.ldraw + h * V + v0 + c] = o;
    }
    __syncthreads();
    if (mine) {
      float u[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[e] = s_u[cg * VEC + e];
#pragma unroll
      for (int i = 0; i < kStepRows; ++i) {
        const int d = rg + i * rpp;
        if (d < D) {
          const float k = s_gqk[d].z;
#pragma unroll
          for (int e = 0; e < VEC; ++e) S[i][e] += k * u[e];
          if (t + 1 == ntok) store_vec<VEC>(sp + static_cast<long long>(d) * V, S[i]);
        }
      }
    }
    if (fused) {
      // the CTA holds the whole head: normalise over the value columns, weigh and gate
      float ss = 0.f;
      for (int c = lane; c < V; c += 32) ss += s_o[c] * s_o[c];
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(V) + a.eps);
      for (int c = tid; c < V; c += kStepThreads) {
        if (c != tid) {                // heads wider than the CTA
          gate = static_cast<float>(static_cast<const T*>(a.gate)[row * a.ldg + h * V + c]);
          weight = norm_w[c];
        }
        static_cast<T*>(a.out)[row * a.ldo + h * V + c] = static_cast<T>(s_o[c] * inv * weight * gate_value(a.gate_kind, gate));
      }
    }
    if (t + 1 < ntok) __syncthreads();   // s_gqk, s_v, s_o are rewritten
  }
}

// Decode steps at full bandwidth: one CTA per (sequence, head), the head's state fetched by one bulk copy into shared memory
// while the token's inputs are prepared (three CTAs per SM, six of half the threads for small states, keep copies in flight),
// updated from there straight back to global memory. One-token segments, whole heads, vdim a multiple of 4.
template <typename T, int MODE, bool CONV, int NT>
__global__ void __launch_bounds__(NT, 3 * kStepThreads / NT)
stream_step_kernel(const DmoeRecur a) {
  constexpr bool DELTA = MODE == kDelta;
  extern __shared__ __align__(128) float s_stream[];
  __shared__ __align__(8) unsigned long long s_bar;
  __shared__ int s_abort;
  const int tid = threadIdx.x, lane = tid & 31;
  const int4 seg = a.segs != nullptr ? static_cast<const int4*>(a.segs)[blockIdx.x] : row_segment(a, blockIdx.x);
  const int slot = seg.z, pos = seg.w, h = blockIdx.y, D = a.dim, V = a.vdim;
  if (seg.y <= 0 || slot < 0 || slot >= a.n_slots) return;
  const long long row = seg.x;
  const int hk = DELTA ? h / (a.heads / a.kv_heads) : h;
  float* s_S = s_stream;                                            // [D][V]
  float4* s_gqk = reinterpret_cast<float4*>(s_S + D * V);        // [D]
  float* s_v = reinterpret_cast<float*>(s_gqk + D);              // [V]
  float* s_red = s_v + V;                                        // [DELTA ? 2 : 1][rpp][V]
  float* s_u = s_v;                                              // column c of v and of the sums is read by the thread
  float* s_o = s_red;                                            // that then writes u and o there
  float* sp = a.state + (static_cast<long long>(slot) * a.heads + h) * D * V;
  const uint32_t bar = smem_u32(&s_bar);
  if (tid == 0) {
    s_abort = 0;
    mbar_init(bar, 1);
    mbar_fence_init();
    if (pos > 0) {
      const uint32_t bytes = static_cast<uint32_t>(D) * V * 4;
      mbar_expect_tx(bar, bytes);
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(s_S)),
                   "l"(sp), "r"(bytes), "r"(bar) : "memory");
    }
  }
  const int vq = V / 4, rpp = NT / vq, cg = tid % vq, rg = tid / vq;
  const bool mine = rg < rpp;
  const float* norm_w = a.norm_w + h * a.norm_ld;
  float beta = 0.f, gate = 0.f, weight = 0.f;
  if (DELTA) beta = static_cast<float>(static_cast<const T*>(a.beta)[row * a.ldb + h]);
  const bool fused = a.raw == nullptr;
  if (fused && tid < V) {
    gate = static_cast<float>(static_cast<const T*>(a.gate)[row * a.ldg + h * V + tid]);
    weight = norm_w[tid];
  }
  TokenGates tg = {};
  if (MODE == kMemory) {
    tg = token_gates(a, row, pos, slot, h);
    if (tid == 0) *max_state(a, slot, pos, h) = tg.top;
  }
  token_inputs<T, MODE, CONV>(a, row, pos, slot, h, hk, 0, V, decay_scale(a, h), tg, s_gqk, s_v);
  __syncthreads();                                               // the inputs, and the barrier's initialisation
  const RowFactors f = row_factors<MODE>(a, s_gqk, tg);
  if (MODE == kMemory && !fused && tid == 0) a.scale[row * a.heads + h] = f.scale;
  if (DELTA) beta = 1.f / (1.f + expf(-beta));
  if (pos > 0 && !mbar_wait(bar, 0, &s_abort) && tid == 0 && a.status != nullptr) atomicExch(a.status, kStatusBarrierTimeout);
  float rq[4] = {0.f, 0.f, 0.f, 0.f}, rk[4] = {0.f, 0.f, 0.f, 0.f};
  if (mine) {
    if (pos > 0) {
#pragma unroll 8
      for (int d = rg; d < D; d += rpp) {
        const float4 x = s_gqk[d];
        const float4 s = *reinterpret_cast<const float4*>(s_S + d * V + cg * 4);
        const float f0 = MODE == kBonus ? 1.f : x.x;
        const float sv[4] = {s.x * f0, s.y * f0, s.z * f0, s.w * f0};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          rq[e] += sv[e] * x.y;
          if (DELTA) rk[e] += sv[e] * x.z;
        }
      }
    }
    store_vec<4>(s_red + rg * V + cg * 4, rq);
    if (DELTA) store_vec<4>(s_red + (rpp + rg) * V + cg * 4, rk);
  }
  __syncthreads();
  if (s_abort) {                                                 // the copy never came: leave state and output alone
    for (int i = 0; i < (1 << 20) && !mbar_try_wait(bar, 0); ++i) {}
    return;
  }
  for (int c = tid; c < V; c += NT) {
    float oq = 0.f, ok = 0.f;
#pragma unroll 4
    for (int r = 0; r < rpp; ++r) {
      oq += s_red[r * V + c];
      if (DELTA) ok += s_red[(rpp + r) * V + c];
    }
    float u = s_v[c];
    if (DELTA) u = beta * (u - ok * f.fk);
    s_u[c] = u * f.fk;
    const float o = oq * f.fq + f.qk * f.fq * f.fk * u;
    if (fused) s_o[c] = o * f.scale;
    else a.raw[row * a.ldraw + h * V + c] = o;
  }
  __syncthreads();
  if (mine) {
    const float4 u = *reinterpret_cast<const float4*>(s_u + cg * 4);
#pragma unroll 8
    for (int d = rg; d < D; d += rpp) {
      const float4 x = s_gqk[d];
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
      if (pos > 0) s = *reinterpret_cast<const float4*>(s_S + d * V + cg * 4);
      *reinterpret_cast<float4*>(sp + static_cast<long long>(d) * V + cg * 4) =
          make_float4(s.x * x.x + x.z * u.x, s.y * x.x + x.z * u.y, s.z * x.x + x.z * u.z, s.w * x.x + x.z * u.w);
    }
  }
  if (!fused) return;
  float ss = 0.f;
  for (int c = lane; c < V; c += 32) ss += s_o[c] * s_o[c];
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(V) + a.eps);
  for (int c = tid; c < V; c += NT) {
    if (c != tid) {                                              // heads wider than the CTA
      gate = static_cast<float>(static_cast<const T*>(a.gate)[row * a.ldg + h * V + c]);
      weight = norm_w[c];
    }
    static_cast<T*>(a.out)[row * a.ldo + h * V + c] = static_cast<T>(s_o[c] * inv * weight * gate_value(a.gate_kind, gate));
  }
}

// out[row, h, :] = raw / sqrt(mean(raw^2) + eps) * norm_w * gate for the rows of a table (segs or chunks; NULL: entry i is
// row i); `lanes` (a power of two) threads per (row, head), VEC consecutive columns per lane and pass
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
gate_norm_kernel(const int4* __restrict__ table, const float* __restrict__ raw, long long ldraw, const T* __restrict__ gate,
                 long long ldg, const float* __restrict__ norm_w, int norm_ld, float eps, int gate_kind, T* __restrict__ out,
                 long long ldo, int heads, int V, int lanes, const float* __restrict__ scale) {
  const int4 e = table != nullptr ? table[blockIdx.x] : make_int4(blockIdx.x, 1, 0, 0);
  const int lane = threadIdx.x & (lanes - 1), per = blockDim.x / lanes;       // (row, head) pairs of the CTA at a time
  const auto sum = [&](float v) {                // over the lanes of a pair; the whole warp takes part
    for (int o = lanes / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
  };
  const int pairs = e.y * heads;
  for (int i0 = blockIdx.y * per; i0 < pairs; i0 += gridDim.y * per) {
    const bool on = i0 + static_cast<int>(threadIdx.x) / lanes < pairs;
    const int i = on ? i0 + threadIdx.x / lanes : pairs - 1;
    const long long row = e.x + i / heads;
    const int h = i % heads;
    const float* r = raw + row * ldraw + h * V;
    const T* gp = gate + row * ldg + h * V;
    const float* nw = norm_w + h * norm_ld;
    const float f = scale != nullptr ? scale[row * heads + h] : 1.f;
    float x[VEC], gv[VEC], w[VEC];
    float ss = 0.f;
    const int c0 = lane * VEC;
    if (c0 < V) {                          // the first pass stays in registers (all of it where V <= 32 VEC)
      load_vec<VEC>(r + c0, x);
      load_any<VEC>(gp + c0, gv);
      load_vec<VEC>(nw + c0, w);
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss += x[k] * x[k];
    }
    for (int c = c0 + lanes * VEC; c < V; c += lanes * VEC) {
      float y[VEC];
      load_vec<VEC>(r + c, y);
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss += y[k] * y[k];
    }
    const float inv = f / sqrtf(sum(ss) * f * f / static_cast<float>(V) + eps);
    for (int c = on ? c0 : V; c < V; c += lanes * VEC) {
      if (c != c0) {
        load_vec<VEC>(r + c, x);
        load_any<VEC>(gp + c, gv);
        load_vec<VEC>(nw + c, w);
      }
#pragma unroll
      for (int k = 0; k < VEC; ++k) x[k] *= inv * w[k] * gate_value(gate_kind, gv[k]);
      store_any<VEC>(out + row * ldo + h * V + c, x);
    }
  }
}

// The same where all heads are normed together: one CTA per row, its first NV * 256 * VEC columns in registers.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
wide_gate_norm_kernel(const int4* __restrict__ table, const float* __restrict__ raw, long long ldraw, const T* __restrict__ gate,
                      long long ldg, const float* __restrict__ norm_w, float eps, int gate_kind, T* __restrict__ out,
                      long long ldo, int V) {
  constexpr int NV = 2;
  __shared__ float s_part[2][8];
  const int4 e = table != nullptr ? table[blockIdx.x] : make_int4(blockIdx.x, 1, 0, 0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int buf = 0;
  for (int t = blockIdx.y; t < e.y; t += gridDim.y, buf ^= 1) {
    const long long row = e.x + t;
    const float* r = raw + row * ldraw;
    float x[NV][VEC], gv[NV][VEC], w[VEC], ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = (k * 256 + threadIdx.x) * VEC;
      if (c < V) {
        load_vec<VEC>(r + c, x[k]);
        load_any<VEC>(gate + row * ldg + c, gv[k]);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss += x[k][i] * x[k][i];
      }
    }
    for (int c = (NV * 256 + threadIdx.x) * VEC; c < V; c += 256 * VEC) {
      float y[VEC];
      load_vec<VEC>(r + c, y);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += y[i] * y[i];
    }
    ss = warp_sum(ss);
    if (lane == 0) s_part[buf][warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) ss += s_part[buf][k];
    const float inv = 1.f / sqrtf(ss / static_cast<float>(V) + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = (k * 256 + threadIdx.x) * VEC;
      if (c < V) {
        load_vec<VEC>(norm_w + c, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[k][i] *= inv * w[i] * gate_value(gate_kind, gv[k][i]);
        store_any<VEC>(out + row * ldo + c, x[k]);
      }
    }
    for (int c = (NV * 256 + threadIdx.x) * VEC; c < V; c += 256 * VEC) {
      float y[VEC], g[VEC];
      load_vec<VEC>(r + c, y);
      load_any<VEC>(gate + row * ldg + c, g);
      load_vec<VEC>(norm_w + c, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] *= inv * w[i] * gate_value(gate_kind, g[i]);
      store_any<VEC>(out + row * ldo + c, y);
    }
  }
}

// Matrix memory, longer segments: log decay, factor of k and running maximum of every token, one CTA per (segment, head), 1024 tokens
// at a time. A run of tokens is a map m -> max(F + m, I); maps are composed along the tokens. Whatever wins the maximum is then a
// sum over few tokens (logs of input gates are bounded), so nothing cancels.
constexpr int kGateThreads = 1024;
__device__ __forceinline__ void scan_max_plus(float& F, float& I, int lane) {       // over the warp, inclusive
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float fl = __shfl_up_sync(0xffffffffu, F, o), il = __shfl_up_sync(0xffffffffu, I, o);
    if (lane >= o) {
      I = fmaxf(il + F, I);
      F += fl;
    }
  }
}
__global__ void __launch_bounds__(kGateThreads) memory_gates_kernel(const DmoeRecur a) {
  __shared__ float s_F[kGateThreads / 32], s_I[kGateThreads / 32], s_top[kGateThreads];
  const int4 seg = static_cast<const int4*>(a.segs)[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, slot = seg.z;
  if (seg.y <= 0 || slot < 0 || slot >= a.n_slots) return;
  float top = seg.w > 0 ? *max_state(a, slot, seg.w - 1, h) : 0.f;       // before the pass
  float i = -INFINITY, f = 0.f;
  if (tid < seg.y) memory_logs(a, seg.x + tid, h, i, f);
  for (int t0 = 0; t0 < seg.y; t0 += kGateThreads) {
    const int t = t0 + tid;
    float ni = -INFINITY, nf = 0.f;
    if (t + kGateThreads < seg.y) memory_logs(a, seg.x + t + kGateThreads, h, ni, nf);
    float F = f, I = i;
    scan_max_plus(F, I, lane);
    if (lane == 31) {
      s_F[warp] = F;
      s_I[warp] = I;
    }
    __syncthreads();
    float wF = s_F[lane], wI = s_I[lane];
    scan_max_plus(wF, wI, lane);
    wF = __shfl_sync(0xffffffffu, wF, max(warp - 1, 0));
    wI = __shfl_sync(0xffffffffu, wI, max(warp - 1, 0));
    const float base = warp > 0 ? fmaxf(wF + top, wI) : top;               // before this warp's tokens
    const float m = fmaxf(F + base, I);
    s_top[tid] = m;
    __syncthreads();
    if (t < seg.y) {
      const float before = tid > 0 ? s_top[tid - 1] : top;
      const long long at = h * a.ldsteps + seg.x + t;
      // the steps are those between the stored maxima, whatever their rounding
      a.keep[at] = f + before - m;
      a.put[at] = expf(i - m);
      a.run_max[at] = m;
      if (t + 1 == seg.y) *max_state(a, slot, seg.w + t, h) = m;
    }
    top = s_top[kGateThreads - 1];
    i = ni;
    f = nf;
    __syncthreads();                                     // s_top and the warps' maps are rewritten
  }
}

// Causal depthwise convolution + silu of the q | k | v projections of one chunk of a segment, VEC neighbouring channels per
// thread (TAPS: bound of the number of taps). The taps before the segment's first row come from the ring: ring[slot][p % taps][channel] = projection at p.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128)
conv_chunk_kernel(const DmoeRecur a, const int4* __restrict__ chunks, T* __restrict__ out, long long ldo) {
  constexpr int HIST = TAPS - 1, STEP = 8;
  const int4 ck = chunks[blockIdx.x];
  const int4 seg = static_cast<const int4*>(a.segs)[ck.z];
  const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= C || seg.z < 0 || seg.z >= a.n_slots) return;
  const int R = a.taps, qc = a.kv_heads * a.dim;
  const T* src;
  long long ld;
  if (c < qc) { src = static_cast<const T*>(a.q) + c; ld = a.ldq; }
  else if (c < 2 * qc) { src = static_cast<const T*>(a.k) + c - qc; ld = a.ldk; }
  else { src = static_cast<const T*>(a.v) + c - 2 * qc; ld = a.ldv; }
  const T* ring = static_cast<const T*>(a.ring) + static_cast<long long>(seg.z) * R * C + c;
  float w[TAPS][VEC];               // w[j]: weight of the input j tokens back
  float x[HIST + STEP][VEC];            // x[HIST + i]: input of row i of the step
  const int pos0 = seg.w + (ck.x - seg.x);     // position of the chunk's first row
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
#pragma unroll
    for (int e = 0; e < VEC; ++e) w[j][e] = j < R ? a.conv_w[static_cast<long long>(c + e) * R + R - 1 - j] : 0.f;
#pragma unroll
  for (int j = 1; j <= HIST; ++j) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[HIST - j][e] = 0.f;
    if (j < R && pos0 - j >= 0)
      load_any<VEC>(ck.x - j >= seg.x ? src + (ck.x - j) * ld : ring + static_cast<long long>((pos0 - j) % R) * C, x[HIST - j]);
  }
  for (int t = 0; t < ck.y; t += STEP) {
#pragma unroll
    for (int i = 0; i < STEP; ++i) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[HIST + i][e] = 0.f;
      if (t + i < ck.y) load_any<VEC>(src + (ck.x + t + i) * ld, x[HIST + i]);
    }
#pragma unroll
    for (int i = 0; i < STEP; ++i) {
      if (t + i < ck.y) {
        float acc[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          acc[e] = 0.f;
#pragma unroll
          for (int j = TAPS - 1; j >= 0; --j) acc[e] += w[j][e] * x[HIST + i - j][e];
          acc[e] = sizeof(T) == 2 ? __fdividef(acc[e], 1.f + __expf(-acc[e])) : silu(acc[e]);
        }
        store_any<VEC>(out + (ck.x + t + i) * ldo + c, acc);
      }
    }
#pragma unroll
    for (int j = 0; j < HIST; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[j][e] = x[STEP + j][e];
  }
}

// Writes the last taps - 1 projections of every segment into the ring (after conv_chunk_kernel has read the old ones).
template <typename T>
__global__ void __launch_bounds__(256) ring_update_kernel(const DmoeRecur a) {
  const int4 seg = static_cast<const int4*>(a.segs)[blockIdx.x];
  const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim, R = a.taps, qc = a.kv_heads * a.dim;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C || seg.z < 0 || seg.z >= a.n_slots) return;
  T* ring = static_cast<T*>(a.ring) + static_cast<long long>(seg.z) * R * C + c;
  for (int j = 1; j < R && j <= seg.y; ++j) {
    const long long row = seg.x + seg.y - j;
    T v;
    if (c < qc) v = static_cast<const T*>(a.q)[row * a.ldq + c];
    else if (c < 2 * qc) v = static_cast<const T*>(a.k)[row * a.ldk + c - qc];
    else v = static_cast<const T*>(a.v)[row * a.ldv + c - 2 * qc];
    ring[static_cast<long long>((seg.w + seg.y - j) % R) * C] = v;
  }
}

static int check_recur(const DmoeRecur* a) {
  if (a->heads < 1 || a->kv_heads < 1 || a->heads % a->kv_heads != 0 || a->dim < 1 || a->vdim < 1) return -10;
  if (a->heads > 65535 || a->state == nullptr || a->n_slots < 1) return -10;
  if (a->decay_kind < 3 ? a->z_bias == nullptr : a->decay_kind == 3 ? a->head_decay == nullptr
                        : a->gates == nullptr || a->gate_bias == nullptr || a->norm_state == nullptr || a->max_state == nullptr) return -10;
  if (a->decay_kind >= 3 && (a->delta || a->bonus != nullptr || a->taps > 0)) return -10;
  if (a->decay_kind == 4 && a->raw != nullptr && a->scale == nullptr) return -10;
  if (a->segs == nullptr && (a->positions == nullptr || a->rows == nullptr || a->kv_slots == nullptr)) return -10;
  if ((a->decay_kind == 1 && a->a_log == nullptr) || (a->bonus != nullptr && (a->delta || a->taps > 0))) return -10;
  if (a->taps < 0 || a->taps > kMaxTaps || (a->taps > 0 && (a->conv_w == nullptr || a->ring == nullptr))) return -11;
  return 0;
}

constexpr int kStreamSmem = 76400;       // three CTAs per SM
constexpr int kSmallState = 32 * 1024;   // states up to here take half the threads, six CTAs per SM

// Shared memory of stream_step_kernel, or 0 where it does not apply: whole heads of a multiple of 4 value columns whose
// state leaves room for three CTAs per SM.
static int stream_threads(const DmoeRecur& a) {
  return a.dim * a.vdim * 4 <= kSmallState && a.vdim <= 2 * kStepThreads ? kStepThreads / 2 : kStepThreads;
}
static size_t stream_smem(const DmoeRecur& a) {
  if (a.vdim % 4 != 0 || a.vdim > 4 * kStepThreads || (reinterpret_cast<uintptr_t>(a.state) & 15) != 0)
    return 0;
  const int rpp = stream_threads(a) / (a.vdim / 4);
  const size_t b = (static_cast<size_t>(a.dim) * a.vdim + 4 * a.dim + a.vdim + static_cast<size_t>(a.delta ? 2 : 1) * rpp * a.vdim) * 4;
  return b <= kStreamSmem ? b : 0;
}

template <typename T, int MODE, bool CONV, int NT>
static int launch_stream_nt(const DmoeRecur& a, size_t smem, cudaStream_t stream) {
  static PerDeviceOnce configured;
  const int rc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(stream_step_kernel<T, MODE, CONV, NT>,
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, kStreamSmem));
  });
  if (rc != 0) return rc;
  return static_cast<int>(launch_kernel(stream_step_kernel<T, MODE, CONV, NT>, dim3(a.n_segs, a.heads), dim3(NT), smem,
                                        stream, a));
}
template <typename T, int MODE, bool CONV>
static int launch_stream(const DmoeRecur& a, size_t smem, cudaStream_t stream) {
  return stream_threads(a) == kStepThreads ? launch_stream_nt<T, MODE, CONV, kStepThreads>(a, smem, stream)
                                           : launch_stream_nt<T, MODE, CONV, kStepThreads / 2>(a, smem, stream);
}

template <typename T, int MODE, bool CONV, int VEC>
static int launch_step(const DmoeRecur& a, int vt, cudaStream_t stream) {
  const int vq = vt / VEC, rpp = kStepThreads / vq;
  const size_t smem = (4 * static_cast<size_t>(a.dim) + 3 * vt + static_cast<size_t>(MODE == kDelta ? 2 : 1) * rpp * vt) * sizeof(float);
  if (smem > 48 * 1024) return -13;
  const dim3 grid(a.n_segs, a.heads, (a.vdim + vt - 1) / vt);
  return static_cast<int>(launch_kernel(step_kernel<T, MODE, CONV, VEC>, grid, dim3(kStepThreads), smem, stream, a, vt));
}

template <typename T>
static int step_dispatch(const DmoeRecur& a, int vt, bool vec, cudaStream_t stream) {
  const bool conv = a.taps > 0;
  const size_t smem = a.one_token && vt >= a.vdim ? stream_smem(a) : 0;
  if (smem > 0) {
    if (a.decay_kind == 4) return launch_stream<T, kMemory, false>(a, smem, stream);
    if (a.bonus != nullptr) return launch_stream<T, kBonus, false>(a, smem, stream);
    if (!a.delta) return conv ? -12 : launch_stream<T, kPlain, false>(a, smem, stream);
    return conv ? launch_stream<T, kDelta, true>(a, smem, stream) : launch_stream<T, kDelta, false>(a, smem, stream);
  }
  if (a.decay_kind == 4)
    return vec ? launch_step<T, kMemory, false, 4>(a, vt, stream) : launch_step<T, kMemory, false, 1>(a, vt, stream);
  if (a.bonus != nullptr)
    return vec ? launch_step<T, kBonus, false, 4>(a, vt, stream) : launch_step<T, kBonus, false, 1>(a, vt, stream);
  if (!a.delta) {
    if (conv) return -12;
    return vec ? launch_step<T, kPlain, false, 4>(a, vt, stream) : launch_step<T, kPlain, false, 1>(a, vt, stream);
  }
  if (conv) return vec ? launch_step<T, kDelta, true, 4>(a, vt, stream) : launch_step<T, kDelta, true, 1>(a, vt, stream);
  return vec ? launch_step<T, kDelta, false, 4>(a, vt, stream) : launch_step<T, kDelta, false, 1>(a, vt, stream);
}

}  // namespace dmoe

using namespace dmoe;

// Largest value tile of a CTA (a multiple of 4 where vectors are used): the state tile must fit the registers.
extern "C" int dmoe_recur_value_tile(int dim, int vdim) {
  const int vec = vdim % 4 == 0 ? 4 : 1;
  int vt = vdim;
  for (;;) {
    const int vq = (vt + vec - 1) / vec;
    if (vq <= kStepThreads && static_cast<long long>(kStepThreads / vq) * kStepRows >= dim) return vq * vec;
    if (vq <= 1) return 0;
    vt = (vq + 1) / 2 * vec;
  }
}

// One launch over all segments of a->segs, token by token. a->taps > 0: q, k, v are raw projections and every segment has
// one token; otherwise they are final. a->raw == NULL (needs vt >= vdim): the gated, normalised rows go to a->out;
// otherwise the read-outs go to a->raw (dmoe_gate_norm finishes them).
extern "C" int dmoe_recur_step(const DmoeRecur* a, int vt, void* stream_) {
  const int rc = check_recur(a);
  if (rc != 0) return rc;
  if (a->n_segs == 0) return 0;
  const bool vec = a->vdim % 4 == 0 && vt % 4 == 0 && (reinterpret_cast<uintptr_t>(a->state) & 15) == 0;
  const int per = vec ? 4 : 1;
  if (a->decay_kind == 4 && !a->one_token && (a->keep == nullptr || a->put == nullptr || a->run_max == nullptr)) return -15;
  if (vt < 1 || vt / per > kStepThreads || static_cast<long long>(kStepThreads / (vt / per)) * kStepRows < a->dim) return -13;
  if (a->raw == nullptr && (vt < a->vdim || a->out == nullptr || a->gate == nullptr || a->norm_w == nullptr)) return -14;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  return a->is_f32 ? step_dispatch<float>(*a, vt, vec, stream) : step_dispatch<__nv_bfloat16>(*a, vt, vec, stream);
}

extern "C" int dmoe_gate_norm(int is_f32, const void* table, int n, int max_tokens, const float* raw, long long ldraw,
                              const void* gate, long long ldg, const float* norm_w, int norm_ld, float eps, int gate_kind, void* out,
                              long long ldo, int heads, int V, const float* scale, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (heads < 1 || V < 1 || max_tokens < 1) return -10;
  if (n == 0) return 0;
  if (heads == 1 && V > 512 && scale == nullptr) {
    const auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool v4 = V % 4 == 0 && ldraw % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && al16(raw) && al16(gate) && al16(out) && al16(norm_w);
    const dim3 g(n, max_tokens < 64 ? max_tokens : 64);
    const int4* tb = static_cast<const int4*>(table);
#define DMOE_WIDE(T_, VEC_)                                                                                                    \
  wide_gate_norm_kernel<T_, VEC_><<<g, 256, 0, stream>>>(tb, raw, ldraw, static_cast<const T_*>(gate), ldg, norm_w, eps, gate_kind, \
                                                         static_cast<T_*>(out), ldo, V)
    if (is_f32 && v4) DMOE_WIDE(float, 4);
    else if (is_f32) DMOE_WIDE(float, 1);
    else if (v4) DMOE_WIDE(__nv_bfloat16, 4);
    else DMOE_WIDE(__nv_bfloat16, 1);
#undef DMOE_WIDE
    return static_cast<int>(cudaGetLastError());
  }
  long long by = (static_cast<long long>(max_tokens) * heads + 31) / 32;     // about four (row, head) pairs per warp
  if (by > 1024) by = 1024;
  const dim3 grid(n, static_cast<unsigned>(by));
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = V % 4 == 0 && norm_ld % 4 == 0 && ldraw % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && al(raw) && al(gate) && al(out) && al(norm_w);
  int lanes = 32;
  while (lanes > 4 && (lanes / 2) * (vec ? 4 : 1) >= V) lanes /= 2;
#define DMOE_GATE_NORM(T_, VEC_)                                                                                       \
  gate_norm_kernel<T_, VEC_><<<grid, 256, 0, stream>>>(static_cast<const int4*>(table), raw, ldraw,                    \
                                                       static_cast<const T_*>(gate), ldg, norm_w, norm_ld, eps, gate_kind, \
                                                       static_cast<T_*>(out), ldo, heads, V, lanes, scale)
  if (is_f32) {
    if (vec) DMOE_GATE_NORM(float, 4);
    else DMOE_GATE_NORM(float, 1);
  } else {
    if (vec) DMOE_GATE_NORM(__nv_bfloat16, 4);
    else DMOE_GATE_NORM(__nv_bfloat16, 1);
  }
#undef DMOE_GATE_NORM
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_memory_gates(const DmoeRecur* a, void* stream) {
  const int rc = check_recur(a);
  if (rc != 0) return rc;
  if (a->decay_kind != 4 || a->segs == nullptr || a->keep == nullptr || a->put == nullptr || a->run_max == nullptr) return -15;
  if (a->n_segs == 0) return 0;
  memory_gates_kernel<<<dim3(a->n_segs, a->heads), kGateThreads, 0, static_cast<cudaStream_t>(stream)>>>(*a);
  return static_cast<int>(cudaGetLastError());
}

// Convolved, activated q | k | v of the chunked segments -> out [rows, ldo]; then the ring takes their last inputs.
extern "C" int dmoe_conv_chunks(const DmoeRecur* a, const void* chunks, int n_chunks, void* out, long long ldo, void* stream_) {
  const int rc = check_recur(a);
  if (rc != 0) return rc;
  if (a->taps < 1) return -11;
  if (n_chunks == 0 || a->n_segs == 0) return 0;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  const int C = 2 * a->kv_heads * a->dim + a->heads * a->vdim;
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 3) == 0; };
  const bool pairs = !a->is_f32 && (a->kv_heads * a->dim) % 2 == 0 && C % 2 == 0 && a->ldq % 2 == 0 && a->ldk % 2 == 0 &&
                     a->ldv % 2 == 0 && ldo % 2 == 0 && al(a->q) && al(a->k) && al(a->v) && al(out) && al(a->ring);
  const int per = pairs ? 256 : 128;
  const dim3 g1(n_chunks, (C + per - 1) / per), g2(a->n_segs, (C + 255) / 256);
  const int4* ck = static_cast<const int4*>(chunks);
#define DMOE_CONV(T_, VEC_)                                                                                       \
  do {                                                                                                           \
    if (a->taps <= 4) conv_chunk_kernel<T_, VEC_, 4><<<g1, 128, 0, stream>>>(*a, ck, static_cast<T_*>(out), ldo); \
    else conv_chunk_kernel<T_, VEC_, kMaxTaps><<<g1, 128, 0, stream>>>(*a, ck, static_cast<T_*>(out), ldo);      \
    ring_update_kernel<T_><<<g2, 256, 0, stream>>>(*a);                                                          \
  } while (0)
  if (a->is_f32) DMOE_CONV(float, 1);
  else if (pairs) DMOE_CONV(__nv_bfloat16, 2);
  else DMOE_CONV(__nv_bfloat16, 1);
#undef DMOE_CONV
  return static_cast<int>(cudaGetLastError());
}
