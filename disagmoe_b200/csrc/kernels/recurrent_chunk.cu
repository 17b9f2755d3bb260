// Chunked form of the linear recurrences of recurrent.cu for prompts: 64 tokens at a time on the tensor cores.
//
// With b_t the running sum of the log decays inside a chunk (per key channel), S_0 the state before it and
// u_j = v_j (plain write) or u = the solution of (I + A) u = beta (v - (k e^b) S_0), A_tj = beta_t sum_d k_t k_j e^(b_t - b_j),
// j < t (delta rule):
//
//   o_t = (q_t e^(b_t)) S_0 + sum_{j <= t} P_tj u_j,   P_tj = sum_d q_t k_j e^(b_t - b_j)
//   S   = e^(b_end) S_0 + sum_j (k_j e^(b_end - b_j)) u_j^T
//
// chunk_prep_kernel computes everything that does not depend on S_0, one CTA per (chunk, head): P, q e^b, k e^(b_end - b)
// and for the delta rule T = (I + A)^-1, W = -T (beta k e^b), U0 = T (beta v), so that u = U0 + W S_0.
// chunk_scan_kernel then walks the chunks of a segment in order, one CTA per (segment, head, value tile), with the state in
// its accumulators.
//
// Precision: decays, their sums and exponentials, unit norms, T and the state are fp32; matrix products split both
// operands into bf16 hi + lo parts and accumulate in fp32 (see mma_sync.cuh). P and A are products of rows scaled by
// e^(b_t - m) and e^(m - b_j), m = b in the middle of the chunk; where a channel decays so fast that these could
// overflow (more than 2^60 either way), the pairwise exponentials are evaluated one by one.
#include "mma_sync.cuh"
#include "recurrent.cuh"

namespace dmoe {

constexpr int kChunk = 64;
constexpr int kChunkThreads = 256;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kMaxShift = 60.f;          // log2 units
constexpr int kMid = 31;
constexpr int kPs = kChunk + 8;            // row stride (elements) of 64-column bf16 tiles in shared memory

// Workspace of one (chunk, head), in bytes.
template <int DP>
struct ChunkWs {
  static constexpr long long kPlane = 2ll * kChunk * DP;          // one bf16 plane [64][DP]
  static constexpr long long kQ = 0, kK = 2 * kPlane, kP = 4 * kPlane, kDec = kP + 4ll * kChunk * kChunk;
  static constexpr long long kW = kDec + 4ll * DP, kU = kW + 2 * kPlane;
  static long long bytes(bool delta, int V) { return delta ? kU + 4ll * kChunk * V : kW; }
};

template <int N>
__device__ __forceinline__ void load_bf16(const __nv_bfloat16* p, float* f) {
  if (N == 4) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    f[0] = x.x; f[N - 3] = x.y; f[N - 2] = y.x; f[N - 1] = y.y;
  } else if (N == 2) {
    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    f[0] = x.x; f[N - 1] = x.y;
  } else {
    f[0] = __bfloat162float(p[0]);
  }
}
// hi / lo planes of N consecutive fp32 values
template <int N>
__device__ __forceinline__ void store_split(__nv_bfloat16* hi, __nv_bfloat16* lo, const float* f) {
  if (N == 1) {
    hi[0] = __float2bfloat16(f[0]);
    lo[0] = __float2bfloat16(bf16_rest(f[0]));
    return;
  }
  uint32_t h[(N + 1) / 2], l[(N + 1) / 2];
#pragma unroll
  for (int i = 0; i < (N + 1) / 2; ++i) split2(f[2 * i], f[2 * i + (N > 1)], h[i], l[i]);
  if (N == 4) {
    *reinterpret_cast<uint2*>(hi) = make_uint2(h[0], h[N / 4]);
    *reinterpret_cast<uint2*>(lo) = make_uint2(l[0], l[N / 4]);
  } else {
    *reinterpret_cast<uint32_t*>(hi) = h[0];
    *reinterpret_cast<uint32_t*>(lo) = l[0];
  }
}

// T = (I + A)^-1 for a strictly lower triangular A [64][65]: 16 x 16 diagonal blocks by forward substitution, then the
// blocks below them, one block diagonal after the other: T_IJ = -T_II sum_{J <= K < I} A_IK T_KJ. `m` is scratch
// [3][16][17]. All 256 threads; T is complete after the last barrier.
__device__ __forceinline__ void invert_unit_lower(const float* A, float* T, float* m) {
  constexpr int LD = kChunk + 1;
  const int tid = threadIdx.x;
  for (int i = tid; i < kChunk * LD; i += kChunkThreads) T[i] = 0.f;
  __syncthreads();
  if (tid < kChunk) {
    const int o = tid / 16 * 16, c = tid % 16;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s = i == c ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) s -= A[(o + i) * LD + o + j] * x[j];
      x[i] = i >= c ? s : 0.f;
      T[(o + i) * LD + o + c] = x[i];
    }
  }
  __syncthreads();
  const int i = tid / 16, j = tid % 16;
  for (int dist = 1; dist < 4; ++dist) {
    for (int I = dist; I < 4; ++I) {
      const int J = I - dist;
      float s = 0.f;
      for (int k = 16 * J; k < 16 * I; ++k) s += A[(16 * I + i) * LD + k] * T[k * LD + 16 * J + j];
      m[(J * 16 + i) * 17 + j] = s;
    }
    __syncthreads();
    for (int I = dist; I < 4; ++I) {
      const int J = I - dist;
      float s = 0.f;
      for (int k = 0; k < 16; ++k) s -= T[(16 * I + i) * LD + 16 * I + k] * m[(J * 16 + k) * 17 + j];
      T[(16 * I + i) * LD + 16 * J + j] = s;
    }
    __syncthreads();
  }
}

template <int DP, bool DELTA>
struct PrepSmem {
  static constexpr int kKs = DP + 8;
  static constexpr int kKn = 2 * kChunk * kKs * 2, kTX = DELTA ? 4 * kChunk * kPs * 2 : 0;
  static constexpr int kRegion = kKn > kTX ? kKn : kTX;
  static constexpr int kBytes = 4 * kChunk * DP + 4 * 4 * kChunk + kRegion + (DELTA ? 2 * 4 * kChunk * (kChunk + 1) : 0) + 16;
};

template <int DP, bool DELTA>
__global__ void __launch_bounds__(kChunkThreads, 2)
chunk_prep_kernel(const DmoeRecur a, const int4* __restrict__ chunks, uint8_t* __restrict__ ws, long long ws_stride, int h0) {
  using L = ChunkWs<DP>;
  using SM = PrepSmem<DP, DELTA>;
  constexpr int PL = DP / 32, KS = DP / 16, LDA = kChunk + 1;
  extern __shared__ __align__(16) uint8_t s_raw[];
  float* s_b = reinterpret_cast<float*>(s_raw);                 // [64][DP] running log2 decay
  float* s_fq = s_b + kChunk * DP;                              // [64] factor of the raw q row
  float* s_fk = s_fq + kChunk;
  float* s_beta = s_fk + kChunk;
  float* s_tot = s_beta + kChunk;                               // [64], unused slack
  uint8_t* region = reinterpret_cast<uint8_t*>(s_tot + kChunk);
  __nv_bfloat16* s_kh = reinterpret_cast<__nv_bfloat16*>(region);          // k e^(m - b), hi then lo plane
  __nv_bfloat16* s_kl = s_kh + kChunk * SM::kKs;
  float* s_A = reinterpret_cast<float*>(region + SM::kRegion);
  float* s_T = s_A + kChunk * LDA;
  (void)s_tot;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int lm_mi = lane >> 3, lm_r = lane & 7;
  const int4 ck = chunks[blockIdx.x];
  const long long row0 = ck.x;
  const int n = ck.y, h = h0 + blockIdx.y, D = a.dim, V = a.vdim;
  const int hk = DELTA ? h / (a.heads / a.kv_heads) : h;
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + row0 * a.ldq + hk * D;
  const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + row0 * a.ldk + hk * D;
  uint8_t* w = ws + (static_cast<long long>(blockIdx.x) * gridDim.y + blockIdx.y) * ws_stride;
  __nv_bfloat16* w_q = reinterpret_cast<__nv_bfloat16*>(w + L::kQ);
  __nv_bfloat16* w_k = reinterpret_cast<__nv_bfloat16*>(w + L::kK);
  __nv_bfloat16* w_p = reinterpret_cast<__nv_bfloat16*>(w + L::kP);

  // ---- log2 decays and their running sums
  {
    const float scale = a.decay_kind == 0 ? a.inv_tau : expf(a.a_log[h]);
    for (int i = tid; i < kChunk * DP; i += kChunkThreads) {
      const int t = i / DP, d = i % DP;
      s_b[i] = t < n && d < D
                   ? kLog2e * log_decay(a.decay_kind, a.z[(row0 + t) * a.ldz + h * D + d] + a.z_bias[h * D + d], scale)
                   : 0.f;
    }
    if (tid < kChunk)
      s_beta[tid] = DELTA && tid < n
                        ? 1.f / (1.f + expf(-__bfloat162float(static_cast<const __nv_bfloat16*>(a.beta)[(row0 + tid) * a.ldb + h])))
                        : 0.f;
    __syncthreads();
    constexpr int NG = kChunkThreads / DP, LEN = kChunk / NG;
    const int d = tid % DP, gi = tid / DP;
    float run = 0.f;
#pragma unroll 8
    for (int t = gi * LEN; t < (gi + 1) * LEN; ++t) {
      run += s_b[t * DP + d];
      s_b[t * DP + d] = run;
    }
    __syncthreads();
    float before = 0.f;
    for (int j = 0; j < gi; ++j) before += s_b[((j + 1) * LEN - 1) * DP + d];
    __syncthreads();
    for (int t = gi * LEN; t < (gi + 1) * LEN; ++t) s_b[t * DP + d] += before;
    __syncthreads();
  }
  bool wide = false;
  if (tid < DP) {
    const float m = s_b[kMid * DP + tid];
    wide = s_b[tid] - m > kMaxShift || m - s_b[(kChunk - 1) * DP + tid] > kMaxShift;
    reinterpret_cast<float*>(w + L::kDec)[tid] = exp2f(s_b[(kChunk - 1) * DP + tid]);
  }
  const bool slow = __syncthreads_or(wide);

  // ---- rows: unit norms, k e^(m - b) to shared memory, q e^b and k e^(b_end - b) to the workspace
  for (int t = warp; t < kChunk; t += kChunkThreads / 32) {
    const int d0 = lane * PL;
    float q[PL], k[PL];
#pragma unroll
    for (int e = 0; e < PL; ++e) q[e] = k[e] = 0.f;
    if (t < n && d0 < D) {
      load_bf16<PL>(qp + t * a.ldq + d0, q);
      load_bf16<PL>(kp + t * a.ldk + d0, k);
    }
    float fq = a.qscale, fk = 1.f;
    if (DELTA) {
      float qq = 0.f, kk = 0.f;
#pragma unroll
      for (int e = 0; e < PL; ++e) { qq += q[e] * q[e]; kk += k[e] * k[e]; }
      fq *= 1.f / sqrtf(warp_sum(qq) + 1e-6f);
      fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
    }
    if (lane == 0) { s_fq[t] = fq; s_fk[t] = fk; }
    float x[PL], y[PL], z[PL];
#pragma unroll
    for (int e = 0; e < PL; ++e) {
      const float b = s_b[t * DP + d0 + e];
      const float kv = k[e] * fk;
      x[e] = kv * exp2f(s_b[kMid * DP + d0 + e] - b);
      y[e] = kv * exp2f(s_b[(kChunk - 1) * DP + d0 + e] - b);
      z[e] = q[e] * fq * exp2f(b);
    }
    if (!slow) store_split<PL>(s_kh + t * SM::kKs + d0, s_kl + t * SM::kKs + d0, x);
    store_split<PL>(w_k + t * DP + d0, w_k + kChunk * DP + t * DP + d0, y);
    store_split<PL>(w_q + t * DP + d0, w_q + kChunk * DP + t * DP + d0, z);
  }
  __syncthreads();

  // ---- P (warps 0-3) and A (warps 4-7)
  if (!slow) {
    const int mi = warp & 3;
    const bool second = warp >= 4;
    if (DELTA || !second) {
      const int r0 = mi * 16 + g, r1 = r0 + 8;
      const __nv_bfloat16* src = second ? kp : qp;
      const long long ld = second ? a.ldk : a.ldq;
      const float f0 = second ? s_fk[r0] : s_fq[r0], f1 = second ? s_fk[r1] : s_fq[r1];
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
      const uint32_t bh = smem_u32(s_kh), bl = smem_u32(s_kl);
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = j & 1 ? r1 : r0, c = ks * 16 + 2 * tq + (j >> 1) * 8;
          float x[2] = {0.f, 0.f};
          if (r < n && c < D) load_bf16<2>(src + r * ld + c, x);
          const float f = j & 1 ? f1 : f0;
          const float2 b = *reinterpret_cast<const float2*>(s_b + r * DP + c);
          const float2 m = *reinterpret_cast<const float2*>(s_b + kMid * DP + c);
          split2(x[0] * f * exp2f(b.x - m.x), x[1] * f * exp2f(b.y - m.y), ah[j], al[j]);
        }
#pragma unroll
        for (int kg = 0; kg < 4; ++kg) {
          if (kg <= mi) {
            const uint32_t off = ((kg * 16 + (lm_mi >> 1) * 8 + lm_r) * SM::kKs + ks * 16 + (lm_mi & 1) * 8) * 2;
            uint32_t h0_, h1_, h2_, h3_, l0_, l1_, l2_, l3_;
            ldmatrix_x4(bh + off, h0_, h1_, h2_, h3_);
            ldmatrix_x4(bl + off, l0_, l1_, l2_, l3_);
            mma_split(acc[2 * kg], ah, al, h0_, h1_, l0_, l1_);
            mma_split(acc[2 * kg + 1], ah, al, h2_, h3_, l2_, l3_);
          }
        }
      }
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const int c = nt * 8 + 2 * tq;
        if (!second) {
          const float v[4] = {c <= r0 ? acc[nt][0] : 0.f, c + 1 <= r0 ? acc[nt][1] : 0.f, c <= r1 ? acc[nt][2] : 0.f,
                              c + 1 <= r1 ? acc[nt][3] : 0.f};
          store_split<2>(w_p + r0 * kChunk + c, w_p + kChunk * kChunk + r0 * kChunk + c, v);
          store_split<2>(w_p + r1 * kChunk + c, w_p + kChunk * kChunk + r1 * kChunk + c, v + 2);
        } else if (DELTA) {
          s_A[r0 * LDA + c] = c < r0 ? acc[nt][0] * s_beta[r0] : 0.f;
          s_A[r0 * LDA + c + 1] = c + 1 < r0 ? acc[nt][1] * s_beta[r0] : 0.f;
          s_A[r1 * LDA + c] = c < r1 ? acc[nt][2] * s_beta[r1] : 0.f;
          s_A[r1 * LDA + c + 1] = c + 1 < r1 ? acc[nt][3] * s_beta[r1] : 0.f;
        }
      }
    }
  } else {
    for (int i = tid; i < kChunk * kChunk; i += kChunkThreads) {
      const int t = i / kChunk, j = i % kChunk;
      float p = 0.f, kk = 0.f;
      if (j <= t && t < n) {
        for (int d = 0; d < D; ++d) {
          const float e = __bfloat162float(kp[j * a.ldk + d]) * s_fk[j] * exp2f(s_b[t * DP + d] - s_b[j * DP + d]);
          p += __bfloat162float(qp[t * a.ldq + d]) * e;
          if (DELTA) kk += __bfloat162float(kp[t * a.ldk + d]) * e;
        }
      }
      const float pv = p * s_fq[t];
      store_split<1>(w_p + i, w_p + kChunk * kChunk + i, &pv);
      if (DELTA) s_A[t * LDA + j] = j < t ? kk * s_fk[t] * s_beta[t] : 0.f;
    }
  }
  if (!DELTA) return;
  __syncthreads();

  // ---- T, then W = -T (beta k e^b) and U0 = T (beta v), 64 columns at a time
  __nv_bfloat16* s_th = reinterpret_cast<__nv_bfloat16*>(region);
  __nv_bfloat16* s_tl = s_th + kChunk * kPs;
  __nv_bfloat16* s_xh = s_tl + kChunk * kPs;
  __nv_bfloat16* s_xl = s_xh + kChunk * kPs;
  invert_unit_lower(s_A, s_T, reinterpret_cast<float*>(s_xh));
  for (int i = tid; i < kChunk * kChunk / 2; i += kChunkThreads) {
    const int t = i / (kChunk / 2), c = i % (kChunk / 2) * 2;
    const float v[2] = {s_T[t * LDA + c], s_T[t * LDA + c + 1]};
    store_split<2>(s_th + t * kPs + c, s_tl + t * kPs + c, v);
  }
  const int nd = (DP + 63) / 64, nv = (V + 63) / 64;
  const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.v) + row0 * a.ldv + h * V;
  __nv_bfloat16* w_w = reinterpret_cast<__nv_bfloat16*>(w + L::kW);
  float* w_u = reinterpret_cast<float*>(w + L::kU);
  const int mi = warp & 3, nh = warp >> 2;
  for (int x = 0; x < nd + nv; ++x) {
    const bool keys = x < nd;
    const int c0 = (keys ? x : x - nd) * 64;
    for (int i = tid; i < kChunk * 32; i += kChunkThreads) {
      const int t = i / 32, c = i % 32 * 2, cc = c0 + c;
      float v[2] = {0.f, 0.f};
      if (t < n && cc < (keys ? D : V)) {
        load_bf16<2>(keys ? kp + t * a.ldk + cc : vp + t * a.ldv + cc, v);
        const float f = keys ? -s_beta[t] * s_fk[t] : s_beta[t];
        v[0] *= f * (keys ? exp2f(s_b[t * DP + cc]) : 1.f);
        v[1] *= f * (keys ? exp2f(s_b[t * DP + cc + 1]) : 1.f);
      }
      store_split<2>(s_xh + t * kPs + c, s_xl + t * kPs + c, v);
    }
    __syncthreads();
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      if (ks <= mi) {                      // T is lower triangular
        const uint32_t ao = ((mi * 16 + (lm_mi & 1) * 8 + lm_r) * kPs + ks * 16 + (lm_mi >> 1) * 8) * 2;
        uint32_t ah[4], al[4];
        ldmatrix_x4(smem_u32(s_th) + ao, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(smem_u32(s_tl) + ao, al[0], al[1], al[2], al[3]);
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          const uint32_t bo = ((ks * 16 + (lm_mi & 1) * 8 + lm_r) * kPs + nh * 32 + p * 16 + (lm_mi >> 1) * 8) * 2;
          uint32_t h0_, h1_, h2_, h3_, l0_, l1_, l2_, l3_;
          ldmatrix_x4_trans(smem_u32(s_xh) + bo, h0_, h1_, h2_, h3_);
          ldmatrix_x4_trans(smem_u32(s_xl) + bo, l0_, l1_, l2_, l3_);
          mma_split(acc[2 * p], ah, al, h0_, h1_, l0_, l1_);
          mma_split(acc[2 * p + 1], ah, al, h2_, h3_, l2_, l3_);
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      const int c = c0 + nh * 32 + nt * 8 + 2 * tq, r0 = mi * 16 + g, r1 = r0 + 8;
      if (keys) {
        if (c < DP) {
          store_split<2>(w_w + r0 * DP + c, w_w + kChunk * DP + r0 * DP + c, acc[nt]);
          store_split<2>(w_w + r1 * DP + c, w_w + kChunk * DP + r1 * DP + c, acc[nt] + 2);
        }
      } else if (c < V) {
        *reinterpret_cast<float2*>(w_u + r0 * V + c) = make_float2(acc[nt][0], acc[nt][1]);
        *reinterpret_cast<float2*>(w_u + r1 * V + c) = make_float2(acc[nt][2], acc[nt][3]);
      }
    }
    __syncthreads();
  }
}

template <int DP, int VT, bool DELTA>
struct ScanSmem {
  static constexpr int kKs = DP + 8, kVs = VT + 8;
  static constexpr int kRows = kChunk * kKs * 2, kPb = kChunk * kPs * 2, kS = DP * kVs * 2, kUb = kChunk * kVs * 2;
  static constexpr int kBytes = (DELTA ? 6 : 4) * kRows + 2 * kPb + 2 * kS + 2 * kUb;
};

// Chunks of one segment in order. Warps 4-7 own 16 rows each of the read-outs, warps 0-3 of u (delta), warps 0 .. DP / 16
// - 1 sixteen key channels each of the state. The tiles of the next chunk are fetched while the current one computes:
// q e^b and W during the state update, k e^(b_end - b) and P (and v) during the products with the old state.
template <int DP, int VT, bool DELTA>
__global__ void __launch_bounds__(kChunkThreads)
chunk_scan_kernel(const DmoeRecur a, const uint8_t* __restrict__ ws, long long ws_stride, int h0, int n_heads) {
  using L = ChunkWs<DP>;
  using SM = ScanSmem<DP, VT, DELTA>;
  constexpr int NT = VT / 8, KS = DP / 16, MT = DP / 16;
  extern __shared__ __align__(16) uint8_t s_raw[];
  const uint32_t s_q = smem_u32(s_raw);                          // planes hi, lo
  const uint32_t s_k = s_q + 2 * SM::kRows;
  const uint32_t s_w = s_k + 2 * SM::kRows;
  const uint32_t s_p = s_w + (DELTA ? 2 : 0) * SM::kRows;
  const uint32_t s_s = s_p + 2 * SM::kPb;
  const uint32_t s_u = s_s + 2 * SM::kS;
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(s_raw + (s_s - s_q));
  __nv_bfloat16* p_u = reinterpret_cast<__nv_bfloat16*>(s_raw + (s_u - s_q));

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int lm_mi = lane >> 3, lm_r = lane & 7;
  const int4* segs = static_cast<const int4*>(a.segs);
  const int4 seg = segs[blockIdx.x];
  const int slot = seg.z;
  if (seg.y <= 0 || slot < 0 || slot >= a.n_slots) return;
  int before = 0;                                                // chunks of the segments before this one
  for (int i = lane; i < blockIdx.x; i += 32) before += (segs[i].y + kChunk - 1) / kChunk;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
  const int nc = (seg.y + kChunk - 1) / kChunk;
  const int hl = blockIdx.y, h = h0 + hl, D = a.dim, V = a.vdim, v0 = blockIdx.z * VT;

  auto base = [&](int c) { return ws + (static_cast<long long>(before + c) * n_heads + hl) * ws_stride; };
  auto copy_rows = [&](uint32_t dst, const uint8_t* src) {       // two planes [64][DP]
    for (int i = tid; i < 2 * kChunk * (DP / 8); i += kChunkThreads) {
      const int r = i / (DP / 8), c = i % (DP / 8);
      cp_async16(dst + r * (SM::kKs * 2) + c * 16, src + i * 16, true);
    }
  };
  auto load_a = [&](int c) {
    copy_rows(s_q, base(c) + L::kQ);
    if (DELTA) copy_rows(s_w, base(c) + L::kW);
  };
  auto load_b = [&](int c) {
    copy_rows(s_k, base(c) + L::kK);
    const uint8_t* src = base(c) + L::kP;
    for (int i = tid; i < 2 * kChunk * 8; i += kChunkThreads)
      cp_async16(s_p + i / 8 * (kPs * 2) + i % 8 * 16, src + i * 16, true);
    if (!DELTA) {                                                // u = v
      const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.v);
      for (int i = tid; i < kChunk * NT; i += kChunkThreads) {
        const int t = i / NT, cc = v0 + i % NT * 8;
        const bool ok = c * kChunk + t < seg.y && cc < V;
        const long long off = ok ? static_cast<long long>(seg.x + c * kChunk + t) * a.ldv + h * V + cc : 0;
        cp_async16(s_u + t * (SM::kVs * 2) + i % NT * 16, vp + off, ok);
      }
    }
  };
  load_a(0);
  cp_async_commit();
  load_b(0);
  cp_async_commit();

  // the state tile: rows d = warp * 16 + g (+ 8), columns v0 + nt * 8 + 2 tq (+ 1)
  float* sp = a.state + (static_cast<long long>(slot) * a.heads + h) * D * V;
  const int d0 = warp * 16 + g, d1 = d0 + 8;
  float sacc[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    sacc[nt][0] = sacc[nt][1] = sacc[nt][2] = sacc[nt][3] = 0.f;
    const int cc = v0 + nt * 8 + 2 * tq;
    if (warp < MT && seg.w > 0 && cc < V) {
      if (d0 < D) { const float2 x = *reinterpret_cast<const float2*>(sp + d0 * V + cc); sacc[nt][0] = x.x; sacc[nt][1] = x.y; }
      if (d1 < D) { const float2 x = *reinterpret_cast<const float2*>(sp + d1 * V + cc); sacc[nt][2] = x.x; sacc[nt][3] = x.y; }
    }
  }
  auto publish = [&] {                                           // state -> hi / lo planes in shared memory
    if (warp < MT) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int o0 = d0 * SM::kVs + nt * 8 + 2 * tq, o1 = d1 * SM::kVs + nt * 8 + 2 * tq;
        store_split<2>(p_s + o0, p_s + DP * SM::kVs + o0, sacc[nt]);
        store_split<2>(p_s + o1, p_s + DP * SM::kVs + o1, sacc[nt] + 2);
      }
    }
  };
  publish();
  cp_async_wait<1>();
  __syncthreads();

  const int mi = warp & 3, r0 = mi * 16 + g, r1 = r0 + 8;
  for (int c = 0; c < nc; ++c) {
    float dec0 = 0.f, dec1 = 0.f;
    if (warp < MT) {
      const float* dp = reinterpret_cast<const float*>(base(c) + L::kDec);
      dec0 = dp[d0];
      dec1 = dp[d1];
    }
    // products with the old state
    float acc[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    if (DELTA && warp < 4) {
      const float* up = reinterpret_cast<const float*>(base(c) + L::kU);
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int cc = v0 + nt * 8 + 2 * tq;
        if (cc < V) {
          const float2 x = *reinterpret_cast<const float2*>(up + r0 * V + cc), y = *reinterpret_cast<const float2*>(up + r1 * V + cc);
          acc[nt][0] = x.x; acc[nt][1] = x.y; acc[nt][2] = y.x; acc[nt][3] = y.y;
        }
      }
    }
    if (DELTA || warp >= 4) {
      const uint32_t src = warp >= 4 ? s_q : s_w;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        const uint32_t ao = ((mi * 16 + (lm_mi & 1) * 8 + lm_r) * SM::kKs + ks * 16 + (lm_mi >> 1) * 8) * 2;
        uint32_t ah[4], al[4];
        ldmatrix_x4(src + ao, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4(src + SM::kRows + ao, al[0], al[1], al[2], al[3]);
#pragma unroll
        for (int p = 0; p < NT / 2; ++p) {
          const uint32_t bo = ((ks * 16 + (lm_mi & 1) * 8 + lm_r) * SM::kVs + p * 16 + (lm_mi >> 1) * 8) * 2;
          uint32_t h0_, h1_, h2_, h3_, l0_, l1_, l2_, l3_;
          ldmatrix_x4_trans(s_s + bo, h0_, h1_, h2_, h3_);
          ldmatrix_x4_trans(s_s + SM::kS + bo, l0_, l1_, l2_, l3_);
          mma_split(acc[2 * p], ah, al, h0_, h1_, l0_, l1_);
          mma_split(acc[2 * p + 1], ah, al, h2_, h3_, l2_, l3_);
        }
      }
    }
    if (DELTA && warp < 4) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int o0 = r0 * SM::kVs + nt * 8 + 2 * tq, o1 = r1 * SM::kVs + nt * 8 + 2 * tq;
        store_split<2>(p_u + o0, p_u + kChunk * SM::kVs + o0, acc[nt]);
        store_split<2>(p_u + o1, p_u + kChunk * SM::kVs + o1, acc[nt] + 2);
      }
    }
    cp_async_wait<0>();
    __syncthreads();
    if (c + 1 < nc) load_a(c + 1);
    cp_async_commit();

    // read-outs: + P u
    if (warp >= 4) {
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks <= mi) {
          const uint32_t ao = ((mi * 16 + (lm_mi & 1) * 8 + lm_r) * kPs + ks * 16 + (lm_mi >> 1) * 8) * 2;
          uint32_t ah[4], al[4];
          ldmatrix_x4(s_p + ao, ah[0], ah[1], ah[2], ah[3]);
          ldmatrix_x4(s_p + SM::kPb + ao, al[0], al[1], al[2], al[3]);
#pragma unroll
          for (int p = 0; p < NT / 2; ++p) {
            const uint32_t bo = ((ks * 16 + (lm_mi & 1) * 8 + lm_r) * SM::kVs + p * 16 + (lm_mi >> 1) * 8) * 2;
            uint32_t h0_, h1_, h2_, h3_;
            ldmatrix_x4_trans(s_u + bo, h0_, h1_, h2_, h3_);
            if (DELTA) {
              uint32_t l0_, l1_, l2_, l3_;
              ldmatrix_x4_trans(s_u + SM::kUb + bo, l0_, l1_, l2_, l3_);
              mma_split(acc[2 * p], ah, al, h0_, h1_, l0_, l1_);
              mma_split(acc[2 * p + 1], ah, al, h2_, h3_, l2_, l3_);
            } else {                                             // v is exact in bf16
              mma_bf16_16816(acc[2 * p], ah, h0_, h1_);
              mma_bf16_16816(acc[2 * p], al, h0_, h1_);
              mma_bf16_16816(acc[2 * p + 1], ah, h2_, h3_);
              mma_bf16_16816(acc[2 * p + 1], al, h2_, h3_);
            }
          }
        }
      }
      const int t0 = c * kChunk + r0, t1 = c * kChunk + r1;
      float* o0 = a.raw + static_cast<long long>(seg.x + t0) * a.ldraw + h * V;
      float* o1 = a.raw + static_cast<long long>(seg.x + t1) * a.ldraw + h * V;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int cc = v0 + nt * 8 + 2 * tq;
        if (cc < V) {
          if (t0 < seg.y) *reinterpret_cast<float2*>(o0 + cc) = make_float2(acc[nt][0], acc[nt][1]);
          if (t1 < seg.y) *reinterpret_cast<float2*>(o1 + cc) = make_float2(acc[nt][2], acc[nt][3]);
        }
      }
    }
    // state: decay, then + (k e^(b_end - b))^T u
    if (warp < MT) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) { sacc[nt][0] *= dec0; sacc[nt][1] *= dec0; sacc[nt][2] *= dec1; sacc[nt][3] *= dec1; }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        const uint32_t ao = ((ks * 16 + (lm_mi >> 1) * 8 + lm_r) * SM::kKs + warp * 16 + (lm_mi & 1) * 8) * 2;
        uint32_t ah[4], al[4];
        ldmatrix_x4_trans(s_k + ao, ah[0], ah[1], ah[2], ah[3]);
        ldmatrix_x4_trans(s_k + SM::kRows + ao, al[0], al[1], al[2], al[3]);
#pragma unroll
        for (int p = 0; p < NT / 2; ++p) {
          const uint32_t bo = ((ks * 16 + (lm_mi & 1) * 8 + lm_r) * SM::kVs + p * 16 + (lm_mi >> 1) * 8) * 2;
          uint32_t h0_, h1_, h2_, h3_;
          ldmatrix_x4_trans(s_u + bo, h0_, h1_, h2_, h3_);
          if (DELTA) {
            uint32_t l0_, l1_, l2_, l3_;
            ldmatrix_x4_trans(s_u + SM::kUb + bo, l0_, l1_, l2_, l3_);
            mma_split(sacc[2 * p], ah, al, h0_, h1_, l0_, l1_);
            mma_split(sacc[2 * p + 1], ah, al, h2_, h3_, l2_, l3_);
          } else {
            mma_bf16_16816(sacc[2 * p], ah, h0_, h1_);
            mma_bf16_16816(sacc[2 * p], al, h0_, h1_);
            mma_bf16_16816(sacc[2 * p + 1], ah, h2_, h3_);
            mma_bf16_16816(sacc[2 * p + 1], al, h2_, h3_);
          }
        }
      }
    }
    publish();
    cp_async_wait<0>();
    __syncthreads();
    if (c + 1 < nc) load_b(c + 1);
    cp_async_commit();
  }
  if (warp < MT) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int cc = v0 + nt * 8 + 2 * tq;
      if (cc < V) {
        if (d0 < D) *reinterpret_cast<float2*>(sp + d0 * V + cc) = make_float2(sacc[nt][0], sacc[nt][1]);
        if (d1 < D) *reinterpret_cast<float2*>(sp + d1 * V + cc) = make_float2(sacc[nt][2], sacc[nt][3]);
      }
    }
  }
}

template <int DP, bool DELTA>
static int launch_prep(const DmoeRecur& a, const void* chunks, int n_chunks, uint8_t* ws, long long stride, int h0, int hn,
                       cudaStream_t stream) {
  using SM = PrepSmem<DP, DELTA>;
  static PerDeviceOnce configured;
  const int rc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(chunk_prep_kernel<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 SM::kBytes));
  });
  if (rc != 0) return rc;
  chunk_prep_kernel<DP, DELTA><<<dim3(n_chunks, hn), kChunkThreads, SM::kBytes, stream>>>(
      a, static_cast<const int4*>(chunks), ws, stride, h0);
  return static_cast<int>(cudaGetLastError());
}

template <int DP, int VT, bool DELTA>
static int launch_scan(const DmoeRecur& a, const uint8_t* ws, long long stride, int h0, int hn, cudaStream_t stream) {
  using SM = ScanSmem<DP, VT, DELTA>;
  static PerDeviceOnce configured;
  const int rc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(chunk_scan_kernel<DP, VT, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 SM::kBytes));
  });
  if (rc != 0) return rc;
  const dim3 grid(a.n_segs, hn, (a.vdim + VT - 1) / VT);
  chunk_scan_kernel<DP, VT, DELTA><<<grid, kChunkThreads, SM::kBytes, stream>>>(a, ws, stride, h0, hn);
  return static_cast<int>(cudaGetLastError());
}

template <int DP, bool DELTA>
static int run_chunks(const DmoeRecur& a, const void* chunks, int n_chunks, uint8_t* ws, long long ws_bytes, cudaStream_t stream) {
  const long long stride = (ChunkWs<DP>::bytes(DELTA, a.vdim) + 127) / 128 * 128;
  long long per = ws_bytes / (stride * n_chunks);               // heads whose chunks fit the workspace at a time
  if (per < 1) return -15;
  if (per > a.heads) per = a.heads;
  // narrower value tiles where the wide ones would leave SMs idle
  const long long wide = static_cast<long long>(a.n_segs) * per * ((a.vdim + 31) / 32);
  const bool narrow = a.vdim <= 16 || wide < device_num_sms();
  for (int h0 = 0; h0 < a.heads; h0 += static_cast<int>(per)) {
    const int hn = a.heads - h0 < per ? a.heads - h0 : static_cast<int>(per);
    int rc = launch_prep<DP, DELTA>(a, chunks, n_chunks, ws, stride, h0, hn, stream);
    if (rc != 0) return rc;
    rc = narrow ? launch_scan<DP, 16, DELTA>(a, ws, stride, h0, hn, stream)
                : launch_scan<DP, 32, DELTA>(a, ws, stride, h0, hn, stream);
    if (rc != 0) return rc;
  }
  return 0;
}

static int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : 128; }

}  // namespace dmoe

using namespace dmoe;

// Can the chunked kernels run this head shape (bf16 activations)?
extern "C" int dmoe_recur_chunk_ok(int dim, int vdim) {
  return dim >= 8 && dim <= 128 && dim % 8 == 0 && vdim >= 8 && vdim % 8 == 0;
}

// Workspace bytes per head of a call with n_chunks chunks.
extern "C" long long dmoe_recur_chunk_bytes(int dim, int vdim, int delta, int n_chunks) {
  const int dp = padded_dim(dim);
  const long long b = dp == 32 ? ChunkWs<32>::bytes(delta, vdim) : dp == 64 ? ChunkWs<64>::bytes(delta, vdim)
                                                                            : ChunkWs<128>::bytes(delta, vdim);
  return (b + 127) / 128 * 128 * n_chunks;
}

// Segments a->segs (any length) by chunks; q, k, v final (after their convolution), read-outs to a->raw. Two launches per
// group of heads that fits the workspace.
extern "C" int dmoe_recur_chunks(const DmoeRecur* a, const void* chunks, int n_chunks, void* ws, long long ws_bytes,
                                 void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (a->is_f32 || a->taps > 0 || !dmoe_recur_chunk_ok(a->dim, a->vdim) || a->raw == nullptr || a->segs == nullptr ||
      a->heads < 1 || a->heads > 65535 || a->kv_heads < 1 || a->heads % a->kv_heads != 0 || a->state == nullptr)
    return -10;
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (a->ldq % 8 != 0 || a->ldk % 8 != 0 || a->ldv % 8 != 0 || a->ldraw % 2 != 0 || !al(a->q) || !al(a->k) || !al(a->v) ||
      !al(ws) || !al(a->state) || !al(a->raw) || (a->decay_kind != 0 && a->a_log == nullptr) || a->z_bias == nullptr)
    return -11;
  if (n_chunks == 0 || a->n_segs == 0) return 0;
  uint8_t* w = static_cast<uint8_t*>(ws);
  const int dp = padded_dim(a->dim);
  if (a->delta) {
    if (dp == 32) return run_chunks<32, true>(*a, chunks, n_chunks, w, ws_bytes, stream);
    if (dp == 64) return run_chunks<64, true>(*a, chunks, n_chunks, w, ws_bytes, stream);
    return run_chunks<128, true>(*a, chunks, n_chunks, w, ws_bytes, stream);
  }
  if (dp == 32) return run_chunks<32, false>(*a, chunks, n_chunks, w, ws_bytes, stream);
  if (dp == 64) return run_chunks<64, false>(*a, chunks, n_chunks, w, ws_bytes, stream);
  return run_chunks<128, false>(*a, chunks, n_chunks, w, ws_bytes, stream);
}
