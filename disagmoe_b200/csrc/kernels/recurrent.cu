// Linear recurrences with a matrix-valued state per head, S [dim, vdim] in fp32, a decay per head and key channel and
// one of two writes per token:
//
//   plain   S <- diag(a) S + k v^T                                 (gated linear attention)
//   delta   S <- diag(a) S;  S <- S + k (beta (v - S^T k))^T       (gated delta rule)
//   o = S^T q, read after the write
//
// States live in slots: slot = block-table row of the sequence, so a sequence's state is found with the same index as
// its KV pages, and a sequence whose first token is in the batch (position 0) starts from zero whatever the slot held.
//
// Work is described by tables that the host builds once per step:
//   segs    int4 {first row, tokens, slot, position of the first token}; a segment = consecutive rows of one sequence
//   chunks  int4 {first row, tokens <= 64, segment, chunk number in the segment}
// Segments of one token (decoding) take step_kernel, which does everything from the raw projections to the gated,
// normalised output in one launch. Longer ones are convolved by conv_chunk_kernel and then run either through the chunked
// tensor-core kernels of recurrent_chunk.cu or, token by token in fp32 arithmetic, through step_kernel.
#include "dmoe_kernels.h"
#include "recurrent.cuh"

namespace dmoe {

constexpr int kStepThreads = 256;
constexpr int kStepRows = 16;        // state rows a thread holds in registers

// One CTA: one segment, one head, `vt` value columns. Threads form a grid of (vt / VEC) column groups x rpp row groups;
// a thread keeps rows rg, rg + rpp, ... of its VEC columns in registers for the whole segment. Per token the read-outs
// of the decayed state at k and at q are reduced together, and o = (a S)^T q + (k.q) u gives the read-out after the
// write without a second pass.
template <typename T, bool DELTA, bool CONV, int VEC>
__global__ void __launch_bounds__(kStepThreads)
step_kernel(const DmoeRecur a, int vt) {
  extern __shared__ float s_mem[];
  const int tid = threadIdx.x, lane = tid & 31;
  const int4 seg = a.segs != nullptr ? static_cast<const int4*>(a.segs)[blockIdx.x] : row_segment(a, blockIdx.x);
  const int row0 = seg.x, ntok = seg.y, slot = seg.z, pos0 = seg.w;
  if (ntok <= 0 || slot < 0 || slot >= a.n_slots) return;
  const int h = blockIdx.y, D = a.dim, V = a.vdim;
  const int hk = DELTA ? h / (a.heads / a.kv_heads) : h;
  const int v0 = blockIdx.z * vt, nv = min(vt, V - v0);
  const int vq = vt / VEC, rpp = kStepThreads / vq;
  const int cg = tid % vq, rg = tid / vq;
  const bool mine = rg < rpp && cg * VEC < nv;
  float* s_q = s_mem;                  // [D]
  float* s_k = s_q + D;                // [D]
  float* s_g = s_k + D;                // [D] decay factors
  float* s_v = s_g + D;                // [vt]
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
  const float decay_scale = a.decay_kind == 0 ? a.inv_tau : expf(a.a_log[h]);

  for (int t = 0; t < ntok; ++t) {
    const long long row = row0 + t;
    const int pos = pos0 + t;
    for (int i = tid; i < D + nv; i += kStepThreads) {
      if (i < D) {
        float q, k;
        if (CONV) {
          q = conv_step<T>(a, row, pos, slot, hk * D + i, a.q, a.ldq, hk * D + i, h % (a.heads / a.kv_heads) == 0 && v0 == 0);
          k = conv_step<T>(a, row, pos, slot, (a.kv_heads + hk) * D + i, a.k, a.ldk, hk * D + i,
                           h % (a.heads / a.kv_heads) == 0 && v0 == 0);
        } else {
          q = static_cast<float>(static_cast<const T*>(a.q)[row * a.ldq + hk * D + i]);
          k = static_cast<float>(static_cast<const T*>(a.k)[row * a.ldk + hk * D + i]);
        }
        s_q[i] = q;
        s_k[i] = k;
        s_g[i] = expf(log_decay(a.decay_kind, a.z[row * a.ldz + h * D + i] + a.z_bias[h * D + i], decay_scale));
      } else {
        const int c = h * V + v0 + i - D;
        s_v[i - D] = CONV ? conv_step<T>(a, row, pos, slot, 2 * a.kv_heads * D + c, a.v, a.ldv, c, true)
                          : static_cast<float>(static_cast<const T*>(a.v)[row * a.ldv + c]);
      }
    }
    __syncthreads();
    // every warp: |q|^2, |k|^2 and q.k of the raw rows
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int d = lane; d < D; d += 32) {
      const float q = s_q[d], k = s_k[d];
      qq += q * q;
      kk += k * k;
      qk += q * k;
    }
    qk = warp_sum(qk);
    float fq = a.qscale, fk = 1.f;     // factors of the raw rows
    if (DELTA) {
      fq *= 1.f / sqrtf(warp_sum(qq) + 1e-6f);
      fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
    }
    float rq[VEC], rk[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) rq[e] = rk[e] = 0.f;
    if (mine) {
#pragma unroll
      for (int i = 0; i < kStepRows; ++i) {
        const int d = rg + i * rpp;
        if (d < D) {
          const float g = s_g[d], q = s_q[d], k = s_k[d];
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            S[i][e] *= g;
            rq[e] += S[i][e] * q;
            if (DELTA) rk[e] += S[i][e] * k;
          }
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        s_red[rg * vt + cg * VEC + e] = rq[e];
        if (DELTA) s_red[(rpp + rg) * vt + cg * VEC + e] = rk[e];
      }
    }
    __syncthreads();
    for (int c = tid; c < nv; c += kStepThreads) {
      float oq = 0.f, ok = 0.f;
      for (int r = 0; r < rpp; ++r) {
        oq += s_red[r * vt + c];
        if (DELTA) ok += s_red[(rpp + r) * vt + c];
      }
      float u = s_v[c];
      if (DELTA) {
        const float beta = 1.f / (1.f + expf(-static_cast<float>(static_cast<const T*>(a.beta)[row * a.ldb + h])));
        u = beta * (u - ok * fk);
      }
      s_u[c] = u * fk;
      const float o = oq * fq + qk * fq * fk * u;
      if (a.raw != nullptr) a.raw[row * a.ldraw + h * V + v0 + c] = o;
      else s_o[c] = o;
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
          const float k = s_k[d];
#pragma unroll
          for (int e = 0; e < VEC; ++e) S[i][e] += k * u[e];
        }
      }
    }
    if (a.raw == nullptr) {
      // the CTA holds the whole head: normalise over the value columns, weigh and gate
      float ss = 0.f;
      for (int c = lane; c < V; c += 32) ss += s_o[c] * s_o[c];
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(V) + a.eps);
      for (int c = tid; c < V; c += kStepThreads) {
        const float g = static_cast<float>(static_cast<const T*>(a.gate)[row * a.ldg + h * V + c]);
        static_cast<T*>(a.out)[row * a.ldo + h * V + c] = static_cast<T>(s_o[c] * inv * a.norm_w[c] * gate_value(a.gate_kind, g));
      }
    }
    if (t + 1 < ntok) __syncthreads();   // s_k, s_v, s_o are rewritten
  }
#pragma unroll
  for (int i = 0; i < kStepRows; ++i) {
    const int d = rg + i * rpp;
    if (mine && d < D) store_vec<VEC>(sp + static_cast<long long>(d) * V, S[i]);
  }
}

// out[row, h, :] = raw / sqrt(mean(raw^2) + eps) * norm_w * gate for the rows of a table (segs or chunks; NULL: entry i is
// row i); one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256)
gate_norm_kernel(const int4* __restrict__ table, const float* __restrict__ raw, long long ldraw, const T* __restrict__ gate,
                 long long ldg, const float* __restrict__ norm_w, float eps, int gate_kind, T* __restrict__ out,
                 long long ldo, int heads, int V) {
  const int4 e = table != nullptr ? table[blockIdx.x] : make_int4(blockIdx.x, 1, 0, 0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  for (int i = blockIdx.y * nw + warp; i < e.y * heads; i += gridDim.y * nw) {
    const long long row = e.x + i / heads;
    const int h = i % heads;
    const float* r = raw + row * ldraw + h * V;
    float ss = 0.f;
    for (int c = lane; c < V; c += 32) ss += r[c] * r[c];
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(V) + eps);
    for (int c = lane; c < V; c += 32)
      out[row * ldo + h * V + c] =
          static_cast<T>(r[c] * inv * norm_w[c] * gate_value(gate_kind, static_cast<float>(gate[row * ldg + h * V + c])));
  }
}

// Causal depthwise convolution + silu of the q | k | v projections of one chunk of a segment. The taps before the
// segment's first row come from the ring: ring[slot][p % taps][channel] = projection at position p.
template <typename T>
__global__ void __launch_bounds__(128)
conv_chunk_kernel(const DmoeRecur a, const int4* __restrict__ chunks, T* __restrict__ out, long long ldo) {
  const int4 ck = chunks[blockIdx.x];
  const int4 seg = static_cast<const int4*>(a.segs)[ck.z];
  const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C || seg.z < 0 || seg.z >= a.n_slots) return;
  const int R = a.taps, qc = a.kv_heads * a.dim;
  const T* src;
  long long ld;
  if (c < qc) { src = static_cast<const T*>(a.q) + c; ld = a.ldq; }
  else if (c < 2 * qc) { src = static_cast<const T*>(a.k) + c - qc; ld = a.ldk; }
  else { src = static_cast<const T*>(a.v) + c - 2 * qc; ld = a.ldv; }
  const T* ring = static_cast<const T*>(a.ring) + static_cast<long long>(seg.z) * R * C + c;
  float w[kMaxTaps], x[kMaxTaps];      // x[j]: input j tokens back
#pragma unroll
  for (int j = 0; j < kMaxTaps; ++j) {
    w[j] = j < R ? a.conv_w[static_cast<long long>(c) * R + R - 1 - j] : 0.f;
    x[j] = 0.f;
  }
  const int pos0 = seg.w + (ck.x - seg.x);     // position of the chunk's first row
#pragma unroll
  for (int j = 1; j < kMaxTaps; ++j) {
    if (j < R && pos0 - j >= 0)
      x[j] = static_cast<float>(ck.x - j >= seg.x ? src[(ck.x - j) * ld] : ring[static_cast<long long>((pos0 - j) % R) * C]);
  }
  for (int t = 0; t < ck.y; ++t) {
    x[0] = static_cast<float>(src[(ck.x + t) * ld]);
    float acc = 0.f;
#pragma unroll
    for (int j = kMaxTaps - 1; j >= 0; --j) acc += w[j] * x[j];
    out[(ck.x + t) * ldo + c] = static_cast<T>(silu(acc));
#pragma unroll
    for (int j = kMaxTaps - 1; j > 0; --j) x[j] = x[j - 1];
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
  if (a->heads > 65535 || a->state == nullptr || a->z_bias == nullptr || a->n_slots < 1) return -10;
  if (a->segs == nullptr && (a->positions == nullptr || a->rows == nullptr || a->kv_slots == nullptr)) return -10;
  if (a->decay_kind != 0 && a->a_log == nullptr) return -10;
  if (a->taps < 0 || a->taps > kMaxTaps || (a->taps > 0 && (a->conv_w == nullptr || a->ring == nullptr))) return -11;
  return 0;
}

template <typename T, bool DELTA, bool CONV, int VEC>
static int launch_step(const DmoeRecur& a, int vt, cudaStream_t stream) {
  const int vq = vt / VEC, rpp = kStepThreads / vq;
  const size_t smem = (3 * static_cast<size_t>(a.dim) + 3 * vt + static_cast<size_t>(DELTA ? 2 : 1) * rpp * vt) * sizeof(float);
  if (smem > 48 * 1024) return -13;
  const dim3 grid(a.n_segs, a.heads, (a.vdim + vt - 1) / vt);
  return static_cast<int>(launch_kernel(step_kernel<T, DELTA, CONV, VEC>, grid, dim3(kStepThreads), smem, stream, a, vt));
}

template <typename T>
static int step_dispatch(const DmoeRecur& a, int vt, bool vec, cudaStream_t stream) {
  const bool conv = a.taps > 0;
  if (!a.delta) {
    if (conv) return -12;
    return vec ? launch_step<T, false, false, 4>(a, vt, stream) : launch_step<T, false, false, 1>(a, vt, stream);
  }
  if (conv) return vec ? launch_step<T, true, true, 4>(a, vt, stream) : launch_step<T, true, true, 1>(a, vt, stream);
  return vec ? launch_step<T, true, false, 4>(a, vt, stream) : launch_step<T, true, false, 1>(a, vt, stream);
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
  if (vt < 1 || vt / per > kStepThreads || static_cast<long long>(kStepThreads / (vt / per)) * kStepRows < a->dim) return -13;
  if (a->raw == nullptr && (vt < a->vdim || a->out == nullptr || a->gate == nullptr || a->norm_w == nullptr)) return -14;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  return a->is_f32 ? step_dispatch<float>(*a, vt, vec, stream) : step_dispatch<__nv_bfloat16>(*a, vt, vec, stream);
}

extern "C" int dmoe_gate_norm(int is_f32, const void* table, int n, int max_tokens, const float* raw, long long ldraw,
                              const void* gate, long long ldg, const float* norm_w, float eps, int gate_kind, void* out,
                              long long ldo, int heads, int V, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (heads < 1 || V < 1 || max_tokens < 1) return -10;
  if (n == 0) return 0;
  long long by = (static_cast<long long>(max_tokens) * heads + 31) / 32;     // about four (row, head) pairs per warp
  if (by > 1024) by = 1024;
  const dim3 grid(n, static_cast<unsigned>(by));
  if (is_f32)
    gate_norm_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const int4*>(table), raw, ldraw,
                                                      static_cast<const float*>(gate), ldg, norm_w, eps, gate_kind,
                                                      static_cast<float*>(out), ldo, heads, V);
  else
    gate_norm_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(
        static_cast<const int4*>(table), raw, ldraw, static_cast<const __nv_bfloat16*>(gate), ldg, norm_w, eps, gate_kind,
        static_cast<__nv_bfloat16*>(out), ldo, heads, V);
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
  const dim3 g1(n_chunks, (C + 127) / 128), g2(a->n_segs, (C + 255) / 256);
  if (a->is_f32) {
    conv_chunk_kernel<float><<<g1, 128, 0, stream>>>(*a, static_cast<const int4*>(chunks), static_cast<float*>(out), ldo);
    ring_update_kernel<float><<<g2, 256, 0, stream>>>(*a);
  } else {
    conv_chunk_kernel<__nv_bfloat16><<<g1, 128, 0, stream>>>(*a, static_cast<const int4*>(chunks),
                                                             static_cast<__nv_bfloat16*>(out), ldo);
    ring_update_kernel<__nv_bfloat16><<<g2, 256, 0, stream>>>(*a);
  }
  return static_cast<int>(cudaGetLastError());
}
