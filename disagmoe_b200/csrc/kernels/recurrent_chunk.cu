// Chunked form of the linear recurrences of recurrent.cu for prompts: 64 tokens at a time on the tensor cores.
//
// With b_t the running sum of the log decays inside a chunk (per key channel), S_0 the state before it and
// u_j = v_j (plain write) or u = the solution of (I + A) u = beta (v - (k e^b) S_0), A_tj = beta_t sum_d k_t k_j e^(b_t - b_j),
// j < t (delta rule):
//
//   o_t = (q_t e^(b_t)) S_0 + sum_{j <= t} P_tj u_j,   P_tj = sum_d q_t k_j e^(b_t - b_j)
//   S   = e^(b_end) S_0 + sum_j (k_j e^(b_end - b_j)) u_j^T
//
// With a bonus the read-out precedes the token's decay and write: b_(t-1) takes the place of b_t in o_t and P_tj, j < t, and
// P_tt = sum_d q_t bonus k_t; the scan is that of the plain write.
//
// chunk_prep_kernel computes everything that does not depend on S_0, one CTA per (chunk, head): P, q e^b, k e^(b_end - b)
// and for the delta rule T = (I + A)^-1, W = -T (beta k e^b), U0 = T (beta v), so that u = U0 + W S_0.
// chunk_scan_kernel then walks the chunks of a segment in order, one CTA per (segment, head, value tile), with the state in
// its accumulators.
//
// Where a head has one decay (constant, or a matrix memory's), b_t is a number: P = (q k^T) e^(b_t - b_j) with the exponent applied to
// the products of the rows as they are, and the factors of q and k are those of their rows (chunk_prep_head_kernel). The normaliser of a
// matrix memory is one more value tile of the scan, whose only column is ones and whose state lies in n; the CTA that has it
// turns n.q into the factor of the read-outs.
//
// Precision: decays, their sums and exponentials, unit norms, T and the state are fp32; matrix products split both
// operands into bf16 hi + lo parts and accumulate in fp32 (see mma_sync.cuh). P and A are products of rows scaled by
// e^(b_t - m) and e^(m - b_j), m = b in the middle of the chunk; where a channel decays so fast that these could
// overflow (more than 2^60 either way), the pairwise exponentials are evaluated one by one. With a bonus (decays are free there
// and often fast) the scale is that of the key's tile of 16 tokens: q e^(b_(t-1) - m) and k e^(m - b_j), m = b at the tile's end,
// are at most 1 but inside the tile itself, so that only 2^100 within 16 tokens is too fast, and then for the tiles on the diagonal.
#include "mma_sync.cuh"
#include "recurrent.cuh"

namespace dmoe {

constexpr int kChunk = 64;
constexpr int kChunkThreads = 256;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kMaxShift = 60.f;          // log2 units
constexpr float kMaxTileShift = 100.f;
constexpr int kMid = 31;
constexpr int kPs = kChunk + 8;            // row stride (elements) of 64-column bf16 tiles in shared memory

// Workspace of one (chunk, head), in bytes. The left operands of the scan's products (q e^b, (k e^(b_end - b))^T, P, W) are
// stored as mma.sync A fragments: per 16 x 16 tile and plane (hi, lo) one uint4 per lane, so that a warp fetches a tile
// with one coalesced 512-byte load straight into registers. Tile order: q, P, W by (row tile, k tile), k by (channel
// tile, token tile); planes innermost.
template <int DP>
struct ChunkWs {
  static constexpr long long kMat = 2ll * 2 * kChunk * DP;        // both planes of a [64][DP] matrix
  static constexpr long long kQ = 0, kK = kMat, kP = 2 * kMat, kDec = kP + 2ll * 2 * kChunk * kChunk;
  static constexpr long long kW = kDec + 4ll * DP, kU = kW + kMat;
  static long long bytes(bool delta, int V) { return delta ? kU + 4ll * kChunk * V : kW; }
};
constexpr int kFrag = 512;                 // bytes of one fragment tile of one plane

__device__ __forceinline__ void store_frag(uint8_t* tile, int lane, const uint32_t (&f)[4]) {
  reinterpret_cast<uint4*>(tile)[lane] = make_uint4(f[0], f[1], f[2], f[3]);
}
// Issued where it stands (not moved towards its use): the scan prefetches the next chunk's fragments with it.
__device__ __forceinline__ void load_frag(const uint8_t* tile, int lane, uint32_t (&f)[4]) {
  asm volatile("ld.global.v4.u32 {%0, %1, %2, %3}, [%4];"
               : "=r"(f[0]), "=r"(f[1]), "=r"(f[2]), "=r"(f[3]) : "l"(tile + lane * 16));
}
// Two neighbouring accumulator tiles (16 x 8 each) as one A fragment, split into planes.
__device__ __forceinline__ void store_acc_frag(uint8_t* tile, int lane, const float* a, const float* b) {
  uint32_t h[4], l[4];
  split2(a[0], a[1], h[0], l[0]);
  split2(a[2], a[3], h[1], l[1]);
  split2(b[0], b[1], h[2], l[2]);
  split2(b[2], b[3], h[3], l[3]);
  store_frag(tile, lane, h);
  store_frag(tile + kFrag, lane, l);
}

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
      for (int K = J; K < I; ++K) {
#pragma unroll
        for (int k = 0; k < 16; ++k) s += A[(16 * I + i) * LD + 16 * K + k] * T[(16 * K + k) * LD + 16 * J + j];
      }
      m[(J * 16 + i) * 17 + j] = s;
    }
    __syncthreads();
    for (int I = dist; I < 4; ++I) {
      const int J = I - dist;
      float s = 0.f;
#pragma unroll
      for (int k = 0; k < 16; ++k) s -= T[(16 * I + i) * LD + 16 * I + k] * m[(J * 16 + k) * 17 + j];
      T[(16 * I + i) * LD + 16 * J + j] = s;
    }
    __syncthreads();
  }
}

template <int DP, int MODE>
struct PrepSmem {
  static constexpr bool DELTA = MODE == kDelta;
  static constexpr int kKs = DP + 8;
  static constexpr int kKn = 2 * kChunk * kKs * 2, kTX = DELTA ? 4 * kChunk * kPs * 2 : 0;
  static constexpr int kRegion = kKn > kTX ? kKn : kTX;
  static constexpr int kBytes = 4 * kChunk * DP + 3 * 4 * kChunk + kRegion + (DELTA ? 2 * 4 * kChunk * (kChunk + 1) : 0) +
                                (MODE == kBonus ? 4 * 4 * DP : 0) + 16;
};

template <int DP, int MODE>
__global__ void __launch_bounds__(kChunkThreads, MODE == kBonus && DP <= 64 ? 3 : 2)
chunk_prep_kernel(const DmoeRecur a, const int4* __restrict__ chunks, uint8_t* __restrict__ ws, long long ws_stride, int h0) {
  using L = ChunkWs<DP>;
  using SM = PrepSmem<DP, MODE>;
  constexpr bool DELTA = MODE == kDelta, BONUS = MODE == kBonus;
  constexpr int PL = DP / 32, KS = DP / 16, MT = DP / 16, LDA = kChunk + 1, ROWS = kChunk / 8;
  extern __shared__ __align__(16) uint8_t s_raw[];
  float* s_b = reinterpret_cast<float*>(s_raw);                 // [64][DP] running log2 decay
  float* s_fq = s_b + kChunk * DP;                              // [64] factors of the raw q and k rows
  float* s_fk = s_fq + kChunk;
  float* s_beta = s_fk + kChunk;                                // delta: write strengths; bonus: P_tt
  uint8_t* region = reinterpret_cast<uint8_t*>(s_beta + kChunk);
  __nv_bfloat16* s_kh = reinterpret_cast<__nv_bfloat16*>(region);          // scaled k rows, hi then lo plane
  __nv_bfloat16* s_kl = s_kh + kChunk * SM::kKs;
  float* s_A = reinterpret_cast<float*>(region + SM::kRegion);
  float* s_T = s_A + kChunk * LDA;
  float* s_step = s_A;                                          // bonus: [4][DP] decay over tile i of 16 tokens

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int lm_mi = lane >> 3, lm_r = lane & 7;
  const int4 ck = chunks[blockIdx.x];
  const long long row0 = ck.x;
  const int n = ck.y, h = h0 + blockIdx.y, D = a.dim, V = a.vdim;
  const int hk = DELTA ? h / (a.heads / a.kv_heads) : h;
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + row0 * a.ldq + hk * D;
  const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + row0 * a.ldk + hk * D;
  uint8_t* w = ws + (static_cast<long long>(blockIdx.x) * gridDim.y + blockIdx.y) * ws_stride;

  // ---- this warp's rows of k (and q, for its norm); loads first, they are used below
  const int t0 = warp * ROWS, d0 = lane * PL;
  float k[ROWS][PL];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
#pragma unroll
    for (int e = 0; e < PL; ++e) k[i][e] = 0.f;
    if (t0 + i < n && d0 < D) load_bf16<PL>(kp + (t0 + i) * a.ldk + d0, k[i]);
  }
  // ---- log2 decays and their running sums; a thread keeps one channel
  {
    constexpr int NG = kChunkThreads / DP, LEN = kChunk / NG;
    const float scale = decay_scale(a, h);
    const int d = tid % DP, gi = tid / DP;
    const float bias = d < D ? a.z_bias[h * D + d] : 0.f;
    const float* zp = a.z + row0 * a.ldz + h * D + d;
    float run = 0.f;
#pragma unroll
    for (int t8 = 0; t8 < LEN; t8 += 8) {
      float z[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int t = gi * LEN + t8 + j;
        z[j] = t < n && d < D ? zp[t * a.ldz] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int t = gi * LEN + t8 + j;
        if (t < n && d < D) run += kLog2e * log_decay(a.decay_kind, z[j] + bias, scale);
        s_b[t * DP + d] = run;
      }
    }
    if (tid < kChunk)
      s_beta[tid] = DELTA && tid < n
                        ? 1.f / (1.f + expf(-__bfloat162float(static_cast<const __nv_bfloat16*>(a.beta)[(row0 + tid) * a.ldb + h])))
                        : 0.f;
    __syncthreads();
    float before = 0.f;
    for (int j = 0; j < gi; ++j) before += s_b[((j + 1) * LEN - 1) * DP + d];
    __syncthreads();
    if (gi > 0) {
#pragma unroll 8
      for (int t = gi * LEN; t < (gi + 1) * LEN; ++t) s_b[t * DP + d] += before;
    }
  }
  // ---- factors of the rows: scale and unit norms; with a bonus the diagonal of P
  if (DELTA || BONUS) {
    float q[ROWS][PL], bonus[PL];
#pragma unroll
    for (int e = 0; e < PL; ++e) bonus[e] = BONUS && d0 < D ? a.bonus[h * D + d0 + e] : 0.f;
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
#pragma unroll
      for (int e = 0; e < PL; ++e) q[i][e] = 0.f;
      if (t0 + i < n && d0 < D) load_bf16<PL>(qp + (t0 + i) * a.ldq + d0, q[i]);
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      float qq = 0.f, kk = 0.f;
      if (BONUS) {
#pragma unroll
        for (int e = 0; e < PL; ++e) qq += q[i][e] * (k[i][e] * bonus[e]);
        qq = warp_sum(qq);
        if (lane == 0) { s_fq[t0 + i] = a.qscale; s_fk[t0 + i] = 1.f; s_beta[t0 + i] = qq * a.qscale; }
        continue;
      }
#pragma unroll
      for (int e = 0; e < PL; ++e) { qq += q[i][e] * q[i][e]; kk += k[i][e] * k[i][e]; }
      const float fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f), fq = a.qscale / sqrtf(warp_sum(qq) + 1e-6f);
      if (lane == 0) { s_fq[t0 + i] = fq; s_fk[t0 + i] = fk; }
#pragma unroll
      for (int e = 0; e < PL; ++e) k[i][e] *= fk;
    }
  } else if (lane < ROWS) {
    s_fq[t0 + lane] = a.qscale;
    s_fk[t0 + lane] = 1.f;
  }
  __syncthreads();
  bool wide = false;
  if (tid < DP) {
    const float m = s_b[kMid * DP + tid];
    if (BONUS) {
      float from = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float end = s_b[(16 * i + 15) * DP + tid];
        wide = wide || from - end > kMaxTileShift;
        s_step[i * DP + tid] = exp2f(end - from);
        from = end;
      }
    } else {
      wide = s_b[tid] - m > kMaxShift || m - s_b[(kChunk - 1) * DP + tid] > kMaxShift;
    }
    reinterpret_cast<float*>(w + L::kDec)[tid] = exp2f(s_b[(kChunk - 1) * DP + tid]);
  }
  const bool slow = __syncthreads_or(wide);

  // ---- k e^(b_end - b): through shared memory into transposed fragments
  auto stage_k = [&] {
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
      store_split<PL>(s_kh + (t0 + i) * SM::kKs + d0, s_kl + (t0 + i) * SM::kKs + d0, k[i]);
  };
  float to_mid[PL];                                  // e^(m - b_end)
  float k_tile[BONUS ? ROWS : 1][PL];                // k e^(b at the end of its tile - b)
#pragma unroll
  for (int e = 0; e < PL; ++e) {
    const float end = s_b[(kChunk - 1) * DP + d0 + e];
    if (BONUS) {
      const float tile = s_b[(warp / 2 * 16 + 15) * DP + d0 + e], rest = exp2f(end - tile);
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        k_tile[BONUS ? i : 0][e] = k[i][e] * exp2f(tile - s_b[(t0 + i) * DP + d0 + e]);
        k[i][e] = k_tile[BONUS ? i : 0][e] * rest;
      }
      continue;
    }
    to_mid[e] = slow ? 0.f : exp2f(s_b[kMid * DP + d0 + e] - end);
#pragma unroll
    for (int i = 0; i < ROWS; ++i) k[i][e] *= exp2f(end - s_b[(t0 + i) * DP + d0 + e]);
  }
  stage_k();
  __syncthreads();
  for (int i = warp; i < MT * 4; i += kChunkThreads / 32) {
    const int mt = i / 4, ks = i % 4;
    const uint32_t off = ((ks * 16 + (lm_mi >> 1) * 8 + lm_r) * SM::kKs + mt * 16 + (lm_mi & 1) * 8) * 2;
    uint32_t f[4];
    ldmatrix_x4_trans(smem_u32(s_kh) + off, f[0], f[1], f[2], f[3]);
    store_frag(w + L::kK + i * 2 * kFrag, lane, f);
    ldmatrix_x4_trans(smem_u32(s_kl) + off, f[0], f[1], f[2], f[3]);
    store_frag(w + L::kK + (i * 2 + 1) * kFrag, lane, f);
  }
  __syncthreads();
  if (BONUS || !slow) {                              // now k e^(m - b): right operand of P and A
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
#pragma unroll
      for (int e = 0; e < PL; ++e) k[i][e] = BONUS ? k_tile[BONUS ? i : 0][e] : k[i][e] * to_mid[e];
    stage_k();
  }
  __syncthreads();

  // ---- P and the fragments of q e^b. With a bonus warp w and w + 4 share the row tile mi: the upper and the lower half of its key
  // tiles. q's scale starts at the end of the warp's first tile and steps down to the others', at last to the chunk's start.
  if (BONUS) {
    const int mi = warp & 3, r0 = mi * 16 + g, r1 = r0 + 8;
    const int top = warp < 4 ? mi : (mi - 1) / 2, low = warp < 4 ? (mi + 1) / 2 : 0;      // key tiles top .. low
    const bool to_start = low == 0;
    const int skip = slow && warp < 4 ? 1 : 0;       // too fast: the diagonal tile is left to the pairwise path below
    const int from = top - skip;                     // tile whose end is the first scale, -1: the chunk's start
    if (warp < 4 || mi > 0) {
      float acc[2][2][4];                            // [top - kg][8-column half]
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][0][e] = acc[i][1][e] = 0.f;
      const uint32_t bh = smem_u32(s_kh), bl = smem_u32(s_kl);
#pragma unroll
      for (int kb = 0; kb < KS; kb += 4) {           // raw values of up to four k tiles in flight
        uint32_t raw[4][4];
#pragma unroll
        for (int kk = 0; kk < 4 && kb + kk < KS; ++kk)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int r = j & 1 ? r1 : r0, c = (kb + kk) * 16 + 2 * tq + (j >> 1) * 8;
            raw[kk][j] = r < n && c < D ? *reinterpret_cast<const uint32_t*>(qp + r * a.ldq + c) : 0u;
          }
#pragma unroll
        for (int kk = 0; kk < 4 && kb + kk < KS; ++kk) {
          const int ks = kb + kk;
          float2 x[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int r = j & 1 ? r1 : r0, c = ks * 16 + 2 * tq + (j >> 1) * 8;
            x[j] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[kk][j]));
            float2 b = make_float2(0.f, 0.f);
            if (r > 0) b = *reinterpret_cast<const float2*>(s_b + (r - 1) * DP + c);
            float2 m = make_float2(0.f, 0.f);
            if (from >= 0) m = *reinterpret_cast<const float2*>(s_b + (16 * from + 15) * DP + c);
            x[j].x *= a.qscale * exp2f(b.x - m.x);
            x[j].y *= a.qscale * exp2f(b.y - m.y);
          }
          uint32_t ah[4], al[4];
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int kg = top - i;
            if (kg < low) break;
            if (i < skip) continue;
#pragma unroll
            for (int j = 0; j < 4; ++j) split2(x[j].x, x[j].y, ah[j], al[j]);
            const uint32_t off = ((kg * 16 + (lm_mi >> 1) * 8 + lm_r) * SM::kKs + ks * 16 + (lm_mi & 1) * 8) * 2;
            uint32_t h0_, h1_, h2_, h3_, l0_, l1_, l2_, l3_;
            ldmatrix_x4(bh + off, h0_, h1_, h2_, h3_);
            ldmatrix_x4(bl + off, l0_, l1_, l2_, l3_);
            mma_split(acc[i][0], ah, al, h0_, h1_, l0_, l1_);
            mma_split(acc[i][1], ah, al, h2_, h3_, l2_, l3_);
            if (kg > low || to_start) {
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                const float2 st = *reinterpret_cast<const float2*>(s_step + kg * DP + ks * 16 + 2 * tq + (j >> 1) * 8);
                x[j].x *= st.x;
                x[j].y *= st.y;
              }
            }
          }
          if (to_start) {
#pragma unroll
            for (int j = 0; j < 4; ++j) split2(x[j].x, x[j].y, ah[j], al[j]);
            store_frag(w + L::kQ + (mi * KS + ks) * 2 * kFrag, lane, ah);
            store_frag(w + L::kQ + ((mi * KS + ks) * 2 + 1) * kFrag, lane, al);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int kg = top - i;
        if (kg < low) break;
        if (i < skip) continue;
        if (kg == mi) {
#pragma unroll
          for (int h8 = 0; h8 < 2; ++h8)
#pragma unroll
            for (int e = 0; e < 4; ++e) {            // strictly below the diagonal, and the bonus on it
              const int r = e < 2 ? r0 : r1, c = kg * 16 + h8 * 8 + 2 * tq + (e & 1);
              acc[i][h8][e] = c < r ? acc[i][h8][e] : c == r ? s_beta[r] : 0.f;
            }
        }
        store_acc_frag(w + L::kP + (mi * 4 + kg) * 2 * kFrag, lane, acc[i][0], acc[i][1]);
      }
    }
  } else {                                           // warps 0-3; A (warps 4-7)
    const int mi = warp & 3;
    const bool second = warp >= 4;
    if (!second || (DELTA && !slow)) {
      const int r0 = mi * 16 + g, r1 = r0 + 8;
      const __nv_bfloat16* src = second ? kp : qp;
      const long long ld = second ? a.ldk : a.ldq;
      const float f0 = second ? s_fk[r0] : s_fq[r0], f1 = second ? s_fk[r1] : s_fq[r1];
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
      const uint32_t bh = smem_u32(s_kh), bl = smem_u32(s_kl);
#pragma unroll
      for (int kb = 0; kb < KS; kb += 4) {           // raw values of up to four k tiles in flight
        uint32_t raw[4][4];
#pragma unroll
        for (int kk = 0; kk < 4 && kb + kk < KS; ++kk)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int r = j & 1 ? r1 : r0, c = (kb + kk) * 16 + 2 * tq + (j >> 1) * 8;
            raw[kk][j] = r < n && c < D ? *reinterpret_cast<const uint32_t*>(src + r * ld + c) : 0u;
          }
#pragma unroll
        for (int kk = 0; kk < 4 && kb + kk < KS; ++kk) {
          const int ks = kb + kk;
          uint32_t ah[4], al[4], zh[4], zl[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int r = j & 1 ? r1 : r0, c = ks * 16 + 2 * tq + (j >> 1) * 8;
            const float f = j & 1 ? f1 : f0;
            float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[kk][j]));
            x.x *= f;
            x.y *= f;
            const float2 b = *reinterpret_cast<const float2*>(s_b + r * DP + c);
            const float2 m = *reinterpret_cast<const float2*>(s_b + kMid * DP + c);
            split2(x.x * exp2f(b.x - m.x), x.y * exp2f(b.y - m.y), ah[j], al[j]);
            if (!second) split2(x.x * exp2f(b.x), x.y * exp2f(b.y), zh[j], zl[j]);
          }
          if (!second) {
            store_frag(w + L::kQ + (mi * KS + ks) * 2 * kFrag, lane, zh);
            store_frag(w + L::kQ + ((mi * KS + ks) * 2 + 1) * kFrag, lane, zl);
          }
          if (slow) continue;
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
      }
      if (!slow) {
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          const int c = nt * 8 + 2 * tq, edge = second ? -1 : 0;        // A is strictly below the diagonal
          if (c > r0 + edge) acc[nt][0] = 0.f;
          if (c + 1 > r0 + edge) acc[nt][1] = 0.f;
          if (c > r1 + edge) acc[nt][2] = 0.f;
          if (c + 1 > r1 + edge) acc[nt][3] = 0.f;
          if (DELTA && second) {
            s_A[r0 * LDA + c] = acc[nt][0] * s_beta[r0];
            s_A[r0 * LDA + c + 1] = acc[nt][1] * s_beta[r0];
            s_A[r1 * LDA + c] = acc[nt][2] * s_beta[r1];
            s_A[r1 * LDA + c + 1] = acc[nt][3] * s_beta[r1];
          }
        }
        if (!second) {
#pragma unroll
          for (int kg = 0; kg < 4; ++kg)
            store_acc_frag(w + L::kP + (mi * 4 + kg) * 2 * kFrag, lane, acc[2 * kg], acc[2 * kg + 1]);
        }
      }
    }
  }
  if (slow) {
    for (int i = tid; i < (BONUS ? kChunk * 16 : kChunk * kChunk); i += kChunkThreads) {
      const int t = BONUS ? i / 16 : i / kChunk, j = BONUS ? i / 256 * 16 + i % 16 : i % kChunk;
      float p = 0.f, kk = 0.f;
      if ((BONUS ? j < t : j <= t) && t < n) {
        const int tr = BONUS ? t - 1 : t;              // place of the read-out
        for (int d = 0; d < D; ++d) {
          const float e = __bfloat162float(kp[j * a.ldk + d]) * s_fk[j] * exp2f(s_b[tr * DP + d] - s_b[j * DP + d]);
          p += __bfloat162float(qp[t * a.ldq + d]) * e;
          if (DELTA) kk += __bfloat162float(kp[t * a.ldk + d]) * e;
        }
      }
      // place of element (t, j) in the fragment tiles
      const float pv = BONUS && j == t ? s_beta[t] : p * s_fq[t];
      const int r = t % 16, c = j % 16;
      __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(w + L::kP + (t / 16 * 4 + j / 16) * 2 * kFrag) +
                         ((r % 8) * 4 + c % 8 / 2) * 8 + ((r >= 8) + 2 * (c >= 8)) * 2 + c % 2;
      store_split<1>(e, e + kFrag / 2, &pv);
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
  const int nd = (DP + 63) / 64, nv = (V + 63) / 64;
  const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.v) + row0 * a.ldv + h * V;
  float* w_u = reinterpret_cast<float*>(w + L::kU);
  const int mi = warp & 3, nh = warp >> 2;
  uint32_t raw[8];                                   // the next 64-column tile of k or v: rows tid / 32 + 8 i
  auto fetch = [&](int x) {
    const bool keys = x < nd;
    const int cc = (keys ? x : x - nd) * 64 + tid % 32 * 2;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = tid / 32 + 8 * i;
      raw[i] = t < n && cc < (keys ? D : V)
                   ? *reinterpret_cast<const uint32_t*>(keys ? kp + t * a.ldk + cc : vp + t * a.ldv + cc) : 0u;
    }
  };
  fetch(0);
  invert_unit_lower(s_A, s_T, reinterpret_cast<float*>(s_xh));
  for (int i = tid; i < kChunk * kChunk / 2; i += kChunkThreads) {
    const int t = i / (kChunk / 2), c = i % (kChunk / 2) * 2;
    const float v[2] = {s_T[t * LDA + c], s_T[t * LDA + c + 1]};
    store_split<2>(s_th + t * kPs + c, s_tl + t * kPs + c, v);
  }
  for (int x = 0; x < nd + nv; ++x) {
    const bool keys = x < nd;
    const int c0 = (keys ? x : x - nd) * 64;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = tid / 32 + 8 * i, c = tid % 32 * 2, cc = c0 + c;
      const float2 r = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[i]));
      float v[2] = {r.x * s_beta[t], r.y * s_beta[t]};
      if (keys) {
        const float f = -s_fk[t];
        v[0] *= cc < DP ? f * exp2f(s_b[t * DP + cc]) : 0.f;
        v[1] *= cc < DP ? f * exp2f(s_b[t * DP + cc + 1]) : 0.f;
      }
      store_split<2>(s_xh + t * kPs + c, s_xl + t * kPs + c, v);
    }
    if (x + 1 < nd + nv) fetch(x + 1);
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
    if (keys) {
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const int ks = (c0 + nh * 32) / 16 + p;      // k tile of W
        if (ks < KS) store_acc_frag(w + L::kW + (mi * KS + ks) * 2 * kFrag, lane, acc[2 * p], acc[2 * p + 1]);
      }
    } else {
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        const int c = c0 + nh * 32 + nt * 8 + 2 * tq, r0 = mi * 16 + g, r1 = r0 + 8;
        if (c < V) {
          *reinterpret_cast<float2*>(w_u + r0 * V + c) = make_float2(acc[nt][0], acc[nt][1]);
          *reinterpret_cast<float2*>(w_u + r1 * V + c) = make_float2(acc[nt][2], acc[nt][3]);
        }
      }
    }
    __syncthreads();
  }
}

// Preparation where a head has one decay. Warps 0-3: P; warps 4-7: the fragments of q e^b and (k e^(b_end - b))^T.
template <int DP, bool MEM>
__global__ void __launch_bounds__(kChunkThreads, 3)
chunk_prep_head_kernel(const DmoeRecur a, const int4* __restrict__ chunks, uint8_t* __restrict__ ws, long long ws_stride, int h0) {
  using L = ChunkWs<DP>;
  constexpr int KS = DP / 16, MT = DP / 16, LD = DP + 8;
  __shared__ __align__(16) __nv_bfloat16 s_q[kChunk * LD], s_k[kChunk * LD];
  __shared__ float s_b[kChunk], s_put[kChunk];                  // running log2 decay; factor of k
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int lm_mi = lane >> 3, lm_r = lane & 7;
  const int4 ck = chunks[blockIdx.x];
  const long long row0 = ck.x;
  const int n = ck.y, h = h0 + blockIdx.y, D = a.dim;
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + row0 * a.ldq + h * D;
  const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + row0 * a.ldk + h * D;
  uint8_t* w = ws + (static_cast<long long>(blockIdx.x) * gridDim.y + blockIdx.y) * ws_stride;
#pragma unroll
  for (int i = tid; i < kChunk * DP / 8; i += kChunkThreads) {
    const int t = i / (DP / 8), c = i % (DP / 8) * 8;
    const bool in = t < n && c < D;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    *reinterpret_cast<uint4*>(s_q + t * LD + c) = in ? *reinterpret_cast<const uint4*>(qp + t * a.ldq + c) : zero;
    *reinterpret_cast<uint4*>(s_k + t * LD + c) = in ? *reinterpret_cast<const uint4*>(kp + t * a.ldk + c) : zero;
  }
  if (warp == 0) {                                               // two neighbouring tokens per lane
    float b[2], p[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      const long long at = h * a.ldsteps + row0 + t;
      b[e] = t < n ? kLog2e * (MEM ? a.keep[at] : a.head_decay[h]) : 0.f;
      p[e] = t < n ? (MEM ? a.put[at] : 1.f) : 0.f;
    }
    float sum = b[0] + b[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += v;
    }
    s_b[2 * lane] = sum - b[1];
    s_b[2 * lane + 1] = sum;
    s_put[2 * lane] = p[0];
    s_put[2 * lane + 1] = p[1];
  }
  __syncthreads();
  const float end = s_b[kChunk - 1];
  if (tid < DP) reinterpret_cast<float*>(w + L::kDec)[tid] = exp2f(end);
  const uint32_t sq = smem_u32(s_q), sk = smem_u32(s_k);
  if (warp < 4) {
    const int mi = warp, r0 = mi * 16 + g, r1 = r0 + 8;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t qa[4];
      ldmatrix_x4(sq + ((mi * 16 + (lm_mi & 1) * 8 + lm_r) * LD + ks * 16 + (lm_mi >> 1) * 8) * 2, qa[0], qa[1], qa[2], qa[3]);
#pragma unroll
      for (int kg = 0; kg < 4; ++kg) {
        if (kg <= mi) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(sk + ((kg * 16 + (lm_mi >> 1) * 8 + lm_r) * LD + ks * 16 + (lm_mi & 1) * 8) * 2, b0, b1, b2, b3);
          mma_bf16_16816(acc[2 * kg], qa, b0, b1);
          mma_bf16_16816(acc[2 * kg + 1], qa, b2, b3);
        }
      }
    }
    const float br0 = s_b[r0], br1 = s_b[r1];
#pragma unroll
    for (int kg = 0; kg < 4; ++kg) {
      if (kg > mi) continue;
#pragma unroll
      for (int h8 = 0; h8 < 2; ++h8)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = e < 2 ? r0 : r1, c = kg * 16 + h8 * 8 + 2 * tq + (e & 1);
          float& v = acc[2 * kg + h8][e];
          v = c <= r ? v * (a.qscale * s_put[c]) * exp2f((e < 2 ? br0 : br1) - s_b[c]) : 0.f;
        }
      store_acc_frag(w + L::kP + (mi * 4 + kg) * 2 * kFrag, lane, acc[2 * kg], acc[2 * kg + 1]);
    }
    return;
  }
  auto scaled = [&](uint8_t* tile, const uint32_t (&x)[4], const float (&f)[4][2]) {
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x[j]));
      split2(v.x * f[j][0], v.y * f[j][1], hi[j], lo[j]);
    }
    store_frag(tile, lane, hi);
    store_frag(tile + kFrag, lane, lo);
  };
  for (int i = warp - 4; i < 4 * KS; i += 4) {                   // q: rows g and g + 8 of tile mi
    const int mi = i / KS, ks = i % KS;
    uint32_t x[4];
    ldmatrix_x4(sq + ((mi * 16 + (lm_mi & 1) * 8 + lm_r) * LD + ks * 16 + (lm_mi >> 1) * 8) * 2, x[0], x[1], x[2], x[3]);
    const float f0 = a.qscale * exp2f(s_b[mi * 16 + g]), f1 = a.qscale * exp2f(s_b[mi * 16 + g + 8]);
    const float f[4][2] = {{f0, f0}, {f1, f1}, {f0, f0}, {f1, f1}};
    scaled(w + L::kQ + i * 2 * kFrag, x, f);
  }
  for (int i = warp - 4; i < MT * 4; i += 4) {                   // k transposed: columns (tokens) 2 tq, + 1, and 8 further
    const int mt = i / 4, ks = i % 4;
    uint32_t x[4];
    ldmatrix_x4_trans(sk + ((ks * 16 + (lm_mi >> 1) * 8 + lm_r) * LD + mt * 16 + (lm_mi & 1) * 8) * 2, x[0], x[1], x[2], x[3]);
    float f[4][2];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = ks * 16 + 2 * tq + (j >> 1) * 8 + e;
        f[j][e] = s_put[t] * exp2f(end - s_b[t]);
      }
    scaled(w + L::kK + i * 2 * kFrag, x, f);
  }
}

// Chunks of one segment in order. Warps 4-7 own 16 rows each of the read-outs, warps 0-3 of u (delta), warps 0 .. DP / 16
// - 1 sixteen key channels each of the state. Left operands come straight from the workspace into registers, fetched half a
// chunk ahead: q e^b and W while the state is updated, (k e^(b_end - b))^T and P while the old state is multiplied. Only
// the state and u, the right operands that every warp shares, go through shared memory.
template <int DP, int VT, int MODE>
__global__ void __launch_bounds__(kChunkThreads, 1)
chunk_scan_kernel(const DmoeRecur a, const uint8_t* __restrict__ ws, long long ws_stride, int h0, int n_heads) {
  using L = ChunkWs<DP>;
  constexpr bool DELTA = MODE == kDelta, MEM = MODE == kMemory;
  constexpr int NT = VT / 8, KS = DP / 16, MT = DP / 16, VS = VT + 8;
  __shared__ __align__(16) __nv_bfloat16 p_s[2][DP * VS];        // state, planes hi / lo
  __shared__ __align__(16) __nv_bfloat16 p_u[DELTA ? 2 : 1][kChunk * VS];
  const uint32_t s_s = smem_u32(p_s), s_u = smem_u32(p_u);
  constexpr uint32_t kSPlane = DP * VS * 2, kUPlane = kChunk * VS * 2;

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
  const int mi = warp & 3, r0 = mi * 16 + g, r1 = r0 + 8;
  const bool ones = MEM && v0 >= V;                              // the value tile of the normaliser
  const bool reads = warp >= 4, updates = warp < MT;
  const int d0 = warp * 16 + g, d1 = d0 + 8;

  auto base = [&](int c) { return ws + (static_cast<long long>(before + c) * n_heads + hl) * ws_stride; };
  uint32_t fa[KS][2][4];                                         // q e^b (warps 4-7) or W (warps 0-3)
  uint32_t fk[4][2][4], fp[4][2][4];
  float u0[NT][4], dec0 = 0.f, dec1 = 0.f;
  uint4 vnext = make_uint4(0u, 0u, 0u, 0u);                      // plain write: this thread's 8 values of the next v tile
  auto fetch_a = [&](int c) {
    if (reads || DELTA) {
      const uint8_t* p = base(c) + (reads ? L::kQ : L::kW) + mi * KS * 2 * kFrag;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        load_frag(p + ks * 2 * kFrag, lane, fa[ks][0]);
        load_frag(p + (ks * 2 + 1) * kFrag, lane, fa[ks][1]);
      }
    }
    if (DELTA && !reads) {
      const float* up = reinterpret_cast<const float*>(base(c) + L::kU);
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int cc = v0 + nt * 8 + 2 * tq;
        float2 x = make_float2(0.f, 0.f), y = x;
        if (cc < V) {
          x = *reinterpret_cast<const float2*>(up + r0 * V + cc);
          y = *reinterpret_cast<const float2*>(up + r1 * V + cc);
        }
        u0[nt][0] = x.x; u0[nt][1] = x.y; u0[nt][2] = y.x; u0[nt][3] = y.y;
      }
    }
  };
  auto fetch_b = [&](int c) {
    if (updates) {
      const uint8_t* p = base(c) + L::kK + warp * 4 * 2 * kFrag;
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        load_frag(p + ks * 2 * kFrag, lane, fk[ks][0]);
        load_frag(p + (ks * 2 + 1) * kFrag, lane, fk[ks][1]);
      }
      const float* dp = reinterpret_cast<const float*>(base(c) + L::kDec);
      dec0 = dp[d0];
      dec1 = dp[d1];
    }
    if (reads) {
      const uint8_t* p = base(c) + L::kP + mi * 4 * 2 * kFrag;
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks <= mi) {
          load_frag(p + ks * 2 * kFrag, lane, fp[ks][0]);
          load_frag(p + (ks * 2 + 1) * kFrag, lane, fp[ks][1]);
        }
      }
    }
  };
  float top0 = 0.f, top1 = 0.f;                                  // normaliser: running maxima of the rows r0 and r1
  auto fetch_v = [&](int c) {
    if (!DELTA && tid < kChunk * NT) {
      const int t = tid / NT, cc = v0 + tid % NT * 8;
      vnext = make_uint4(0u, 0u, 0u, 0u);
      if (ones) {
        if (c * kChunk + t < seg.y && tid % NT == 0) vnext.x = 0x3f80u;          // bf16 1, 0
      } else if (c * kChunk + t < seg.y && cc < V)
        vnext = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.v) +
                                                static_cast<long long>(seg.x + c * kChunk + t) * a.ldv + h * V + cc);
    }
  };
  auto fetch_top = [&](int c) {
    if (MEM && ones && reads && tq == 0) {
      const float* p = a.run_max + h * a.ldsteps + seg.x + c * kChunk;
      if (c * kChunk + r0 < seg.y) top0 = p[r0];
      if (c * kChunk + r1 < seg.y) top1 = p[r1];
    }
  };
  fetch_a(0);
  fetch_b(0);
  fetch_v(0);
  fetch_top(0);

  // the state tile: rows d = warp * 16 + g (+ 8), columns v0 + nt * 8 + 2 tq (+ 1)
  float* sp = a.state + (static_cast<long long>(slot) * a.heads + h) * D * V;
  float* np = MEM ? a.norm_state + (static_cast<long long>(slot) * a.heads + h) * D : nullptr;
  float sacc[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    sacc[nt][0] = sacc[nt][1] = sacc[nt][2] = sacc[nt][3] = 0.f;
    const int cc = v0 + nt * 8 + 2 * tq;
    if (ones && updates && seg.w > 0 && nt == 0 && tq == 0) {
      if (d0 < D) sacc[nt][0] = np[d0];
      if (d1 < D) sacc[nt][2] = np[d1];
    }
    if (updates && seg.w > 0 && cc < V) {
      if (d0 < D) { const float2 x = *reinterpret_cast<const float2*>(sp + d0 * V + cc); sacc[nt][0] = x.x; sacc[nt][1] = x.y; }
      if (d1 < D) { const float2 x = *reinterpret_cast<const float2*>(sp + d1 * V + cc); sacc[nt][2] = x.x; sacc[nt][3] = x.y; }
    }
  }
  auto publish = [&] {                                           // state -> hi / lo planes in shared memory
    if (updates) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int o0 = d0 * VS + nt * 8 + 2 * tq, o1 = d1 * VS + nt * 8 + 2 * tq;
        store_split<2>(p_s[0] + o0, p_s[1] + o0, sacc[nt]);
        store_split<2>(p_s[0] + o1, p_s[1] + o1, sacc[nt] + 2);
      }
    }
  };
  publish();
  __syncthreads();

  for (int c = 0; c < nc; ++c) {
    if (!DELTA && tid < kChunk * NT) {                           // u = v
      *reinterpret_cast<uint4*>(p_u[0] + tid / NT * VS + tid % NT * 8) = vnext;
      if (c + 1 < nc) fetch_v(c + 1);
    }
    // products with the old state; hi hi and the cross terms in separate accumulators (shorter dependency chains)
    float acc[NT][4], cross[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        acc[nt][e] = DELTA && !reads ? u0[nt][e] : 0.f;
        cross[nt][e] = 0.f;
      }
    if (DELTA || reads) {
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
        for (int p = 0; p < NT / 2; ++p) {
          const uint32_t bo = ((ks * 16 + (lm_mi & 1) * 8 + lm_r) * VS + p * 16 + (lm_mi >> 1) * 8) * 2;
          uint32_t h0_, h1_, h2_, h3_, l0_, l1_, l2_, l3_;
          ldmatrix_x4_trans(s_s + bo, h0_, h1_, h2_, h3_);
          ldmatrix_x4_trans(s_s + kSPlane + bo, l0_, l1_, l2_, l3_);
          mma_bf16_16816(acc[2 * p], fa[ks][0], h0_, h1_);
          mma_bf16_16816(acc[2 * p + 1], fa[ks][0], h2_, h3_);
          mma_bf16_16816(cross[2 * p], fa[ks][0], l0_, l1_);
          mma_bf16_16816(cross[2 * p + 1], fa[ks][0], l2_, l3_);
          mma_bf16_16816(cross[2 * p], fa[ks][1], h0_, h1_);
          mma_bf16_16816(cross[2 * p + 1], fa[ks][1], h2_, h3_);
        }
      }
    }
    if (c + 1 < nc) fetch_a(c + 1);
    if (DELTA && !reads) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] += cross[nt][e];
        const int o0 = r0 * VS + nt * 8 + 2 * tq, o1 = r1 * VS + nt * 8 + 2 * tq;
        store_split<2>(p_u[0] + o0, p_u[DELTA ? 1 : 0] + o0, acc[nt]);
        store_split<2>(p_u[0] + o1, p_u[DELTA ? 1 : 0] + o1, acc[nt] + 2);
      }
    }
    __syncthreads();

    // state: decay, then + (k e^(b_end - b))^T u; read-outs: + P u
    if (updates) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) { sacc[nt][0] *= dec0; sacc[nt][1] *= dec0; sacc[nt][2] *= dec1; sacc[nt][3] *= dec1; }
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
#pragma unroll
      for (int p = 0; p < NT / 2; ++p) {
        const uint32_t bo = ((ks * 16 + (lm_mi & 1) * 8 + lm_r) * VS + p * 16 + (lm_mi >> 1) * 8) * 2;
        uint32_t h0_, h1_, h2_, h3_, l0_ = 0u, l1_ = 0u, l2_ = 0u, l3_ = 0u;
        ldmatrix_x4_trans(s_u + bo, h0_, h1_, h2_, h3_);
        if (DELTA) ldmatrix_x4_trans(s_u + kUPlane + bo, l0_, l1_, l2_, l3_);   // (v is exact in bf16)
        if (updates) {
          mma_bf16_16816(sacc[2 * p], fk[ks][0], h0_, h1_);
          mma_bf16_16816(sacc[2 * p + 1], fk[ks][0], h2_, h3_);
          mma_bf16_16816(sacc[2 * p], fk[ks][1], h0_, h1_);
          mma_bf16_16816(sacc[2 * p + 1], fk[ks][1], h2_, h3_);
          if (DELTA) {
            mma_bf16_16816(sacc[2 * p], fk[ks][0], l0_, l1_);
            mma_bf16_16816(sacc[2 * p + 1], fk[ks][0], l2_, l3_);
          }
        }
        if (reads && ks <= mi) {
          mma_bf16_16816(acc[2 * p], fp[ks][0], h0_, h1_);
          mma_bf16_16816(acc[2 * p + 1], fp[ks][0], h2_, h3_);
          mma_bf16_16816(cross[2 * p], fp[ks][1], h0_, h1_);
          mma_bf16_16816(cross[2 * p + 1], fp[ks][1], h2_, h3_);
          if (DELTA) {
            mma_bf16_16816(cross[2 * p], fp[ks][0], l0_, l1_);
            mma_bf16_16816(cross[2 * p + 1], fp[ks][0], l2_, l3_);
          }
        }
      }
    }
    if (c + 1 < nc) fetch_b(c + 1);
    publish();
    if (reads) {
      const int t0 = c * kChunk + r0, t1 = c * kChunk + r1;
      if (ones && tq == 0) {
        float* sc = a.scale + static_cast<long long>(seg.x) * a.heads + h;
        if (t0 < seg.y) sc[static_cast<long long>(t0) * a.heads] = memory_scale(acc[0][0] + cross[0][0], top0);
        if (t1 < seg.y) sc[static_cast<long long>(t1) * a.heads] = memory_scale(acc[0][2] + cross[0][2], top1);
        if (c + 1 < nc) fetch_top(c + 1);
      }
      float* o0 = a.raw + static_cast<long long>(seg.x + t0) * a.ldraw + h * V;
      float* o1 = a.raw + static_cast<long long>(seg.x + t1) * a.ldraw + h * V;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int cc = v0 + nt * 8 + 2 * tq;
        if (cc < V) {
          if (t0 < seg.y) *reinterpret_cast<float2*>(o0 + cc) = make_float2(acc[nt][0] + cross[nt][0], acc[nt][1] + cross[nt][1]);
          if (t1 < seg.y) *reinterpret_cast<float2*>(o1 + cc) = make_float2(acc[nt][2] + cross[nt][2], acc[nt][3] + cross[nt][3]);
        }
      }
    }
    __syncthreads();
  }
  if (updates) {
    if (ones && tq == 0) {
      if (d0 < D) np[d0] = sacc[0][0];
      if (d1 < D) np[d1] = sacc[0][2];
    }
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

template <int DP, int MODE>
static int launch_prep(const DmoeRecur& a, const void* chunks, int n_chunks, uint8_t* ws, long long stride, int h0, int hn,
                       cudaStream_t stream) {
  using SM = PrepSmem<DP, MODE>;
  static PerDeviceOnce configured;
  const int rc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(chunk_prep_kernel<DP, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 SM::kBytes));
  });
  if (rc != 0) return rc;
  chunk_prep_kernel<DP, MODE><<<dim3(n_chunks, hn), kChunkThreads, SM::kBytes, stream>>>(
      a, static_cast<const int4*>(chunks), ws, stride, h0);
  return static_cast<int>(cudaGetLastError());
}

template <int DP, bool MEM>
static int launch_prep_head(const DmoeRecur& a, const void* chunks, int n_chunks, uint8_t* ws, long long stride, int h0, int hn,
                            cudaStream_t stream) {
  chunk_prep_head_kernel<DP, MEM><<<dim3(n_chunks, hn), kChunkThreads, 0, stream>>>(a, static_cast<const int4*>(chunks), ws, stride, h0);
  return static_cast<int>(cudaGetLastError());
}

template <int DP, int VT, int MODE>
static int launch_scan(const DmoeRecur& a, const uint8_t* ws, long long stride, int h0, int hn, cudaStream_t stream) {
  const dim3 grid(a.n_segs, hn, (a.vdim + VT - 1) / VT + (MODE == kMemory ? 1 : 0));
  chunk_scan_kernel<DP, VT, MODE><<<grid, kChunkThreads, 0, stream>>>(a, ws, stride, h0, hn);
  return static_cast<int>(cudaGetLastError());
}

template <int DP, int MODE>
static int run_chunks(const DmoeRecur& a, const void* chunks, int n_chunks, uint8_t* ws, long long ws_bytes, cudaStream_t stream) {
  constexpr bool DELTA = MODE == kDelta;
  const long long stride = (ChunkWs<DP>::bytes(DELTA, a.vdim) + 127) / 128 * 128;
  long long per = ws_bytes / (stride * n_chunks);               // heads whose chunks fit the workspace at a time
  if (per < 1) return -15;
  if (per > a.heads) per = a.heads;
  // narrower value tiles where the wide ones would leave SMs idle
  const long long wide = static_cast<long long>(a.n_segs) * per * ((a.vdim + 31) / 32);
  const bool narrow = a.vdim <= 16 || wide < device_num_sms();
  for (int h0 = 0; h0 < a.heads; h0 += static_cast<int>(per)) {
    const int hn = a.heads - h0 < per ? a.heads - h0 : static_cast<int>(per);
    int rc;
    if constexpr (MODE == kMemory) rc = launch_prep_head<DP, true>(a, chunks, n_chunks, ws, stride, h0, hn, stream);
    else if (MODE == kPlain && a.decay_kind == 3) rc = launch_prep_head<DP, false>(a, chunks, n_chunks, ws, stride, h0, hn, stream);
    else rc = launch_prep<DP, MODE>(a, chunks, n_chunks, ws, stride, h0, hn, stream);
    if (rc != 0) return rc;
    // the scan of a bonus is that of the plain write
    constexpr int SCAN = MODE == kBonus ? kPlain : MODE;
    rc = narrow ? launch_scan<DP, 16, SCAN>(a, ws, stride, h0, hn, stream)
                : launch_scan<DP, 32, SCAN>(a, ws, stride, h0, hn, stream);
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
      !al(ws) || !al(a->state) || !al(a->raw) || (a->decay_kind == 1 && a->a_log == nullptr) || (a->decay_kind < 3 && a->z_bias == nullptr) || (a->bonus != nullptr && a->delta))
    return -11;
  if (a->decay_kind == 3 && a->head_decay == nullptr) return -11;
  if (a->decay_kind == 4 && (a->keep == nullptr || a->put == nullptr || a->run_max == nullptr || a->scale == nullptr ||
                             a->norm_state == nullptr)) return -11;
  if (a->decay_kind >= 3 && (a->delta || a->bonus != nullptr || a->kv_heads != a->heads)) return -11;
  if (n_chunks == 0 || a->n_segs == 0) return 0;
  uint8_t* w = static_cast<uint8_t*>(ws);
  const int dp = padded_dim(a->dim);
#define DMOE_CHUNKS(MODE_)                                                                     \
  if (dp == 32) return run_chunks<32, MODE_>(*a, chunks, n_chunks, w, ws_bytes, stream);       \
  if (dp == 64) return run_chunks<64, MODE_>(*a, chunks, n_chunks, w, ws_bytes, stream);       \
  return run_chunks<128, MODE_>(*a, chunks, n_chunks, w, ws_bytes, stream)
  if (a->decay_kind == 4) { DMOE_CHUNKS(kMemory); }
  if (a->bonus != nullptr) { DMOE_CHUNKS(kBonus); }
  if (a->delta) { DMOE_CHUNKS(kDelta); }
  DMOE_CHUNKS(kPlain);
#undef DMOE_CHUNKS
}
