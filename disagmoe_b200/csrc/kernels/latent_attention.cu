// Latent attention for sm_100a: keys and values of all heads are linear maps of one cached latent vector per token, plus one
// rotated key part that the heads share. Cache row = [latent (rankp) | rotated key part (rotp)], bf16 (fp32 in
// fp32 runs), rows an odd number of 16-byte units apart.
//
//   latent_prep_kernel     norm of the latent, rotations, cache append, queries head by head for the rows below
//   latent_attn_kernel     rows on their own (decoding, short portions): the key map is already multiplied into the query, so
//                          all heads attend over the cached rows themselves (key = the row, value = its first rankp columns)
//   latent_gather_kernel   cached rows of a prompt run's visible keys, packed for the GEMM that expands them to heads
//   latent_prefill_kernel  prompt runs: causal attention over expanded keys and values
#include "dmoe_kernels.h"
#include "mma_sync.cuh"

namespace dmoe {

typedef __nv_bfloat16 bf16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int pad8(int n) { return (n + 7) / 8 * 8; }

// One CTA per row. A row of y is [heads x (dimp | rotp) | rankp | rotp], parts padded with zeros to multiples of 8.
// VEC: the rotation is interleaved, covers all of rotp and moves in 16-byte units. gate (NULL: none): a row has one gate per head;
// the sigmoid of a loose row's gates becomes the weight of its heads' records.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
latent_prep_kernel(T* __restrict__ y, long long ld, const int* __restrict__ positions, const long long* __restrict__ slots,
                   T* __restrict__ cache, int heads, int dimp, int rotp, int rank, int rankp, int row, int rot,
                   int interleaved, const float2* __restrict__ table, int max_pos, const float* __restrict__ norm_w, float eps,
                   const int* __restrict__ loose, int n_loose, T* __restrict__ xq, T* __restrict__ qa,
                   const T* __restrict__ gate, int4* __restrict__ recs) {
  __shared__ float red[8];
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int half = rot / 2, qd = dimp + rotp;
  const int pos = min(max(positions[t], 0), max_pos - 1);
  const long long slot = slots[t];
  const int li = loose != nullptr ? loose[t] : static_cast<int>(t);
  const float2* tab = table + static_cast<long long>(pos) * half;
  T* yr = y + t * ld;
  const T* c = yr + static_cast<long long>(heads) * qd;

  if (gate != nullptr && li >= 0)
    for (int h = threadIdx.x; h < heads; h += blockDim.x)
      recs[static_cast<long long>(h) * n_loose + li].z = __float_as_int(1.f / (1.f + expf(-static_cast<float>(gate[t * ld + h]))));

  // rotated part of a head (or of the key): pairs turn, what is not rotated passes
  auto turn = [&](const T* p, T* dst, int first, int step) {
    for (int i = first; i < half; i += step) {
      const int a = interleaved ? 2 * i : i, b = interleaved ? 2 * i + 1 : i + half;
      const float u = static_cast<float>(p[a]), v = static_cast<float>(p[b]);
      const float2 cs = tab[i];
      dst[a] = static_cast<T>(u * cs.x - v * cs.y);
      dst[b] = static_cast<T>(v * cs.x + u * cs.y);
    }
    if (p != dst)
      for (int d = rot + first; d < rotp; d += step) dst[d] = p[d];
  };

  if (slot >= 0) {
    float ss = 0.f;
    for (int d = threadIdx.x; d < rank; d += blockDim.x) {
      const float x = static_cast<float>(c[d]);
      ss += x * x;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) ss += red[w];
    const float inv = 1.f / sqrtf(ss / static_cast<float>(rank) + eps);
    T* dst = cache + slot * row;
    for (int d = threadIdx.x; d < rank; d += blockDim.x) dst[d] = static_cast<T>(static_cast<float>(c[d]) * inv * norm_w[d]);
    turn(c + rankp, dst + rankp, threadIdx.x, blockDim.x);
  }
  if (VEC) {
    // units of all heads dealt out to the threads: what is copied, what turns in place and what turns on its way out
    constexpr int V = 16 / sizeof(T);
    const int un = dimp / V, ur = rotp / V, first = li < 0 ? un : 0;
    for (int x = threadIdx.x; x < heads * (un + ur - first); x += blockDim.x) {
      const int h = x / (un + ur - first), u = first + x % (un + ur - first);
      const long long at = static_cast<long long>(h) * n_loose + li;
      T* src = yr + static_cast<long long>(h) * qd + u * V;
      if (u < un) {
        *reinterpret_cast<uint4*>(xq + at * dimp + u * V) = *reinterpret_cast<const uint4*>(src);
        continue;
      }
      alignas(16) T v[V];
      *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(src);
#pragma unroll
      for (int e = 0; e < V / 2; ++e) {
        const float2 cs = tab[(u - un) * (V / 2) + e];
        const float p = static_cast<float>(v[2 * e]), w = static_cast<float>(v[2 * e + 1]);
        v[2 * e] = static_cast<T>(p * cs.x - w * cs.y);
        v[2 * e + 1] = static_cast<T>(w * cs.x + p * cs.y);
      }
      T* dst = li < 0 ? src : qa + at * row + rankp + (u - un) * V;
      *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(v);
    }
    return;
  }
  for (int h = warp; h < heads; h += blockDim.x >> 5) {
    T* q = yr + static_cast<long long>(h) * qd;
    if (li < 0) {
      turn(q + dimp, q + dimp, lane, 32);
      continue;
    }
    const long long at = static_cast<long long>(h) * n_loose + li;
    constexpr int V = 16 / sizeof(T);
    const uint4* src = reinterpret_cast<const uint4*>(q);
    uint4* dst = reinterpret_cast<uint4*>(xq + at * dimp);
    for (int v = lane; v < dimp / V; v += 32) dst[v] = src[v];
    turn(q + dimp, qa + at * row + rankp, lane, 32);
  }
}

__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, const int* __restrict__ block_tables, int max_blocks,
                     const int2* __restrict__ keys, int n, int block_size, int units, uint4* __restrict__ out) {
  const int lane = threadIdx.x & 31;
  const long long i = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (i >= n) return;
  const int2 k = keys[i];
  const long long slot = static_cast<long long>(block_tables[static_cast<long long>(k.x) * max_blocks + k.y / block_size]) * block_size + k.y % block_size;
  for (int v = lane; v < units; v += 32) out[i * units + v] = cache[slot * units + v];
}

// ---------------------------------------------------------------------------------------------------------------------------
// Attention over the cached rows. A CTA (one per SM) has one query token and one range of keys, which a producer warp brings 32
// at a time, one bulk copy per 16 cached rows (consecutive in their page), into a ring of up to 8 tiles. Two groups of eight warps
// consume them with a softmax state and accumulators of their own: up to 16 heads (the rows of the MMA tiles) take turns with the
// tiles and merge at the end; of more heads each group has 16 and sees every tile. Per tile a warp computes the scores of its
// group's heads with 8 keys over one half of the row (S = Q K^T) and leaves them in shared memory; after the tile's only barrier
// every warp takes the whole 16 x 32 score tile back as its own A fragments, does the online softmax (all the same one) and
// accumulates 8 NT value columns (O += P V, V = the same rows, P = hi + lo bf16).
// Cached rows are an odd number of 16-byte units apart, so that ldmatrix meets no bank twice although they are copied as they are.
constexpr int kLatKeys = 32, kLatPiece = 16, kLatThreads = 512 + 32, kLatMaxSmem = 226 * 1024, kLatMaxStages = 8;
constexpr int kLatSp = kLatKeys + 8;        // pitch of a score row, floats: 64-bit reads of a fragment meet no bank twice
constexpr int kLatScores = 2 * 16 * kLatSp; // of one tile: two halves of the row x 16 heads

struct LatentSmem {      // bytes
  int qpitch, stages, q, s, bars, total;
};
__host__ __device__ inline LatentSmem latent_smem(int kd, int row) {
  LatentSmem s;
  s.qpitch = (kd + 31) / 32 * 64 + 16;
  const int fixed = 32 * s.qpitch + 4 * kLatScores * 4 + 16 * kLatMaxStages, fit = (kLatMaxSmem - fixed) / (kLatKeys * row * 2);
  s.stages = fit > kLatMaxStages ? kLatMaxStages : fit;
  s.q = s.stages * kLatKeys * row * 2;
  s.s = s.q + 32 * s.qpitch;
  s.bars = s.s + 4 * kLatScores * 4;
  s.total = s.bars + 16 * kLatMaxStages;
  return s;
}
// Barrier of the 256 threads of a group; true for all of them where `flag` is set for one.
__device__ __forceinline__ bool group_sync_or(int id, bool flag) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbarrier.cta.red.or.pred q, %2, 256, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"(flag ? 1u : 0u), "r"(id) : "memory");
  return r != 0;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// NT: 8-column tiles of the output per warp (rankp <= 64 NT). kd: key size; row: elements from one cached row (or query) to the next.
template <int NT>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_attn_kernel(const bf16* __restrict__ q, const bf16* __restrict__ cache, const int* __restrict__ block_tables,
                   int max_blocks, const int* __restrict__ bt_row, const int* __restrict__ rows, const int* __restrict__ ctx_len,
                   int block_size, int n, int heads, int groups, int rankp, int kd, int row, float scale_log2, int window,
                   const float* __restrict__ sink, int splits, bf16* __restrict__ out, float* __restrict__ part_o,
                   float* __restrict__ part_lse, int* __restrict__ status) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ int s_abort;
  const LatentSmem L = latent_smem(kd, row);
  const int pitch = row * 2;
  const bool both = heads > 16;         // both groups see every tile, 16 heads each
  // the head groups of a token are neighbours: they read the same rows at about the same time
  const int i = blockIdx.x / groups, cta_h0 = blockIdx.x % groups * (both ? 32 : 16), split = blockIdx.y;
  const int warp = threadIdx.x >> 5 & 7, grp = threadIdx.x >> 8, lane = threadIdx.x & 31;   // warp within its group; 2: producer
  const int g = lane >> 2, tq = lane & 3;
  const int b = rows != nullptr ? rows[i] : i;
  const int len = ctx_len[b];
  const int* bt = block_tables + static_cast<long long>(bt_row != nullptr ? bt_row[b] : b) * max_blocks;
  const int lo = window > 0 ? max(0, len - window) : 0, first = lo / kLatPiece * kLatPiece;
  const int per = ((len - first + splits - 1) / splits + kLatKeys - 1) / kLatKeys * kLatKeys;
  const int c0 = min(len, first + split * per), c1 = min(len, c0 + per);
  const int ntile = (c1 - c0 + kLatKeys - 1) / kLatKeys;
  const int k32 = (kd + 31) / 32, khalf = (k32 + 1) / 2;
  const uint32_t sb = smem_u32(smem), full = sb + L.bars, empty = full + 8 * kLatMaxStages;

  if (threadIdx.x == 0) {
    s_abort = 0;
    for (int x = 0; x < L.stages; ++x) {
      mbar_init(full + 8 * x, 1);
      mbar_init(empty + 8 * x, both ? 16 : 8);
    }
    mbar_fence_init();
  }
  // queries, zeros behind them and for absent heads; zeros for rows that neither the last tile nor one before it brings
  for (int x = threadIdx.x; x < (both ? 32 : 16) * (k32 * 4); x += kLatThreads) {
    const int r = x / (k32 * 4), c = x % (k32 * 4);
    const bf16* src = q + (static_cast<long long>(cta_h0 + r) * n + i) * row + c * 8;
    *reinterpret_cast<uint4*>(smem + L.q + r * L.qpitch + c * 16) =
        cta_h0 + r < heads && c * 8 < kd ? *reinterpret_cast<const uint4*>(src) : make_uint4(0, 0, 0, 0);
  }
  if (ntile > 0 && ntile <= L.stages) {
    const int have = c1 - c0 - (ntile - 1) * kLatKeys;
    uint4* z = reinterpret_cast<uint4*>(smem + ((ntile - 1) * kLatKeys + have) * pitch);
    for (int x = threadIdx.x; x < (kLatKeys - have) * (row / 8); x += kLatThreads) z[x] = make_uint4(0, 0, 0, 0);
  }
  __syncthreads();

  float o[NT][4];
#pragma unroll
  for (int x = 0; x < NT; ++x) o[x][0] = o[x][1] = o[x][2] = o[x][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int col0 = warp * NT * 8;                         // this warp's value columns
  bool gave_up = false;
  if (grp == 2) {
    // producer: lane 0 and 1 have a piece of every tile
    for (int j = 0; j < ntile; ++j) {
      const int st = j % L.stages, key = c0 + j * kLatKeys + lane * kLatPiece;
      const int have = lane < 2 ? min(kLatPiece, c1 - key) : 0;
      long long slot = 0;
      if (have > 0) slot = static_cast<long long>(bt[key / block_size]) * block_size + key % block_size;
      if (j >= L.stages) gave_up = !mbar_wait(empty + 8 * st, (j / L.stages - 1) & 1, &s_abort);
      if (__any_sync(0xffffffffu, gave_up)) { gave_up = true; break; }
      if (lane == 0) mbar_expect_tx(full + 8 * st, min(kLatKeys, c1 - key) * pitch);
      __syncwarp();
      if (have > 0)
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                         sb + (st * kLatKeys + lane * kLatPiece) * pitch), "l"(cache + slot * row), "r"(have * pitch),
                     "r"(full + 8 * st) : "memory");
    }
  } else {
    // [group][its tile & 1][half of the row][16][kLatSp] partial scores
    float* s_s = reinterpret_cast<float*>(smem + L.s) + grp * 2 * kLatScores;
    const int lm_mi = lane >> 3, lm_r = lane & 7;
    const int kt = warp & 3, kh = warp >> 2;              // its 8 keys and its half of the row in S
    const int ks0 = kh * khalf, ks1 = min(k32, ks0 + khalf);
    const uint32_t qaddr = sb + L.q + (both ? grp * 16 * L.qpitch : 0) + (lm_r + (lm_mi & 1) * 8) * L.qpitch + (lm_mi >> 1) * 16;
    int buf = 0;
    for (int j = both ? 0 : grp; j < ntile; j += both ? 1 : 2) {
      const int st = j % L.stages;
      const bool ok = mbar_wait(full + st * 8, j / L.stages & 1, &s_abort);
      const uint32_t kb = sb + st * kLatKeys * pitch;
      float* sj = s_s + buf * kLatScores;
      buf ^= 1;
      {
        float s[2][4] = {};
        const uint32_t kaddr = kb + (kt * 8 + lm_r) * pitch + lm_mi * 16;
#pragma unroll 3
        for (int k = ks0; k < ks1; ++k) {
          uint32_t b0, b1, b2, b3, a0[4], a1[4];
          ldmatrix_x4(kaddr + k * 64, b0, b1, b2, b3);
          ldmatrix_x4(qaddr + k * 64, a0[0], a0[1], a0[2], a0[3]);
          ldmatrix_x4(qaddr + k * 64 + 32, a1[0], a1[1], a1[2], a1[3]);
          if (k * 32 + 32 > kd) {       // what lies behind a key is not part of it
            if (k * 32 + 8 >= kd) b1 = 0u;
            if (k * 32 + 16 >= kd) b2 = 0u;
            if (k * 32 + 24 >= kd) b3 = 0u;
          }
          mma_bf16_16816(s[0], a0, b0, b1);
          mma_bf16_16816(s[1], a1, b2, b3);
        }
        float* dst = sj + (kh * 16 + g) * kLatSp + kt * 8 + 2 * tq;
        *reinterpret_cast<float2*>(dst) = make_float2(s[0][0] + s[1][0], s[0][1] + s[1][1]);
        *reinterpret_cast<float2*>(dst + 8 * kLatSp) = make_float2(s[0][2] + s[1][2], s[0][3] + s[1][3]);
      }
      gave_up = group_sync_or(1 + grp, !ok);
      if (gave_up) break;
      if (col0 < rankp) {
        float p[2][8];                  // rows g, g + 8; columns 8 y + 2 tq + {0, 1}, y = 0 .. 3
        const int key = c0 + j * kLatKeys + 2 * tq, seen = c1 - key, from = lo - key;      // visible: from <= column < seen
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float* src = sj + (g + 8 * e) * kLatSp + 2 * tq;
          float mx = m[e];
#pragma unroll
          for (int y = 0; y < 4; ++y) {
            const float2 v = *reinterpret_cast<const float2*>(src + 8 * y);
            const float2 w = *reinterpret_cast<const float2*>(src + 16 * kLatSp + 8 * y);
            p[e][2 * y] = 8 * y < seen && 8 * y >= from ? (v.x + w.x) * scale_log2 : -INFINITY;
            p[e][2 * y + 1] = 8 * y + 1 < seen && 8 * y + 1 >= from ? (v.y + w.y) * scale_log2 : -INFINITY;
            mx = fmaxf(mx, fmaxf(p[e][2 * y], p[e][2 * y + 1]));
          }
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));      // finite: every tile has a visible key
          const float corr = ex2(m[e] - mx);
          m[e] = mx;
          float sum = 0.f;
#pragma unroll
          for (int y = 0; y < 8; ++y) {
            p[e][y] = ex2(p[e][y] - mx);
            sum += p[e][y];
          }
          l[e] = l[e] * corr + sum;     // of this lane's keys; the four lanes of a row add up at the end
#pragma unroll
          for (int x = 0; x < NT; ++x) { o[x][2 * e] *= corr; o[x][2 * e + 1] *= corr; }
        }
#pragma unroll
        for (int ks = 0; ks < kLatKeys / 16; ++ks) {
          uint32_t ph[4], pl[4];
          split2(p[0][4 * ks], p[0][4 * ks + 1], ph[0], pl[0]);
          split2(p[1][4 * ks], p[1][4 * ks + 1], ph[1], pl[1]);
          split2(p[0][4 * ks + 2], p[0][4 * ks + 3], ph[2], pl[2]);
          split2(p[1][4 * ks + 2], p[1][4 * ks + 3], ph[3], pl[3]);
          const uint32_t va = kb + (ks * 16 + (lm_mi & 1) * 8 + lm_r) * pitch + col0 * 2 + (lm_mi >> 1) * 16;
#pragma unroll
          for (int dp = 0; dp < NT / 2; ++dp) {
            if (col0 + dp * 16 < rankp) {
              uint32_t b0, b1, b2, b3;
              ldmatrix_x4_trans(va + dp * 32, b0, b1, b2, b3);
              mma_bf16_16816(o[2 * dp], ph, b0, b1);
              mma_bf16_16816(o[2 * dp + 1], ph, b2, b3);
              mma_bf16_16816(o[2 * dp], pl, b0, b1);
              mma_bf16_16816(o[2 * dp + 1], pl, b2, b3);
            }
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(empty + 8 * st);
    }
  }
  if (__syncthreads_or(gave_up)) {
    // copies may be in flight: give every barrier a last, bounded chance
    if (threadIdx.x == 0 && status != nullptr) atomicExch(status, kStatusBarrierTimeout);
    for (int p = 0; p < L.stages; ++p)
      for (int x = 0; x < (1 << 20) && !(mbar_try_wait(full + 8 * p, 0) && mbar_try_wait(full + 8 * p, 1)); ++x) {}
    return;
  }
  // heads that took turns: the second group leaves its state where the ring was, [16][m, sum], then accumulators as
  // [warp][value][lane]
  float* s_ml = reinterpret_cast<float*>(smem);
  float* s_o = s_ml + 32 + warp * (NT * 4 * 32) + lane;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
  }
  if (grp == 1 && !both) {
    if (warp == 0 && tq == 0) {
      s_ml[2 * g] = m[0]; s_ml[2 * g + 1] = l[0];
      s_ml[2 * (g + 8)] = m[1]; s_ml[2 * (g + 8) + 1] = l[1];
    }
#pragma unroll
    for (int x = 0; x < NT; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) s_o[(x * 4 + e) * 32] = o[x][e];
  }
  __syncthreads();
  if (grp == 2 || (grp == 1 && !both) || col0 >= rankp) return;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int head = cta_h0 + (both ? grp * 16 : 0) + g + 8 * e;
    if (head >= heads) continue;
    const float m1 = both ? -INFINITY : s_ml[2 * (g + 8 * e)], l1 = both ? 0.f : s_ml[2 * (g + 8 * e) + 1];
    const bool sunk = sink != nullptr && split == 0 && len > 0;      // one split carries the sink
    const float sk = sunk ? sink[head] * kLog2e : -INFINITY;
    const float mm = fmaxf(fmaxf(m[e], m1), sk);
    float f0 = 0.f, f1 = 0.f, den = 0.f;
    if (mm > -INFINITY) {
      f0 = exp2f(m[e] - mm);
      f1 = exp2f(m1 - mm);
      den = l[e] * f0 + l1 * f1 + (sunk ? exp2f(sk - mm) : 0.f);
      f0 /= den;
      f1 /= den;
    }
    const long long at = static_cast<long long>(head) * n + i;
#pragma unroll
    for (int x = 0; x < NT; ++x) {
      const int col = col0 + x * 8 + 2 * tq;
      if (col >= rankp) continue;
      float a = o[x][2 * e] * f0, c = o[x][2 * e + 1] * f0;
      if (!both) {
        a += s_o[(x * 4 + 2 * e) * 32] * f1;
        c += s_o[(x * 4 + 2 * e + 1) * 32] * f1;
      }
      if (splits == 1) *reinterpret_cast<uint32_t*>(out + at * rankp + col) = pack_bf16(a, c);
      else *reinterpret_cast<float2*>(part_o + (at * splits + split) * rankp + col) = make_float2(a, c);
    }
    if (splits > 1 && warp == 0 && tq == 0) part_lse[at * splits + split] = den > 0.f ? mm + log2f(den) : -INFINITY;
  }
}

// out[at] = sum over splits of its softmax(lse)-weighted parts, at = (head, query)
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse, int splits, int rankp,
                    bf16* __restrict__ out) {
  const long long at = blockIdx.x;
  float M = -INFINITY;
  for (int s = 0; s < splits; ++s) M = fmaxf(M, part_lse[at * splits + s]);
  float L = 0.f;
  if (M > -INFINITY)
    for (int s = 0; s < splits; ++s) L += exp2f(part_lse[at * splits + s] - M);
  const float inv = L > 0.f ? 1.f / L : 0.f;
  for (int d = threadIdx.x * 2; d < rankp; d += blockDim.x * 2) {
    float x = 0.f, y = 0.f;
    if (L > 0.f)
      for (int s = 0; s < splits; ++s) {
        const float w = exp2f(part_lse[at * splits + s] - M);
        if (w == 0.f) continue;
        const float2 v = *reinterpret_cast<const float2*>(part_o + (at * splits + s) * rankp + d);
        x += w * v.x;
        y += w * v.y;
      }
    *reinterpret_cast<uint32_t*>(out + at * rankp + d) = pack_bf16(x * inv, y * inv);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Prompt runs over expanded keys and values: a CTA of four warps has 64 consecutive tokens of one head (16 per warp as MMA
// rows), keys 64 at a time, double buffered. KD / VD: key (unrotated + rotated) and value sizes rounded up to the tile's.
constexpr int kLpKeys = 64;

template <int KD, int VD>
__global__ void __launch_bounds__(128)
latent_prefill_kernel(const bf16* __restrict__ q, long long ld_q, const bf16* __restrict__ kv, long long ld_kv,
                      const bf16* __restrict__ lat, long long ld_lat, const int4* __restrict__ tiles, const int* __restrict__ base,
                      int dimp, int rotp, int rankp, int vdimp, float scale_log2, int window, const float* __restrict__ sink,
                      const bf16* __restrict__ gate, long long ld_gate, bf16* __restrict__ out, long long ld_out) {
  constexpr int KP = KD * 2 + 16, VP = VD * 2 + 16;       // row pitches: odd numbers of 16-byte units
  constexpr int STAGE = kLpKeys * (KP + VP);
  constexpr int KS = KD / 16, NT = VD / 8;
  extern __shared__ __align__(128) uint8_t smem[];
  const int4 tile = tiles[blockIdx.x];
  const int row0 = tile.x, ntok = tile.y, pos0 = tile.w, head = blockIdx.y;
  const long long kbase = base[blockIdx.x];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tq = lane & 3;
  const int kmax = pos0 + ntok, klo = window > 0 ? max(0, pos0 - window + 1) : 0;
  const int kb0 = klo / kLpKeys, nkb = (kmax + kLpKeys - 1) / kLpKeys;
  const int qd = dimp + rotp, hw = dimp + vdimp;
  const uint32_t sbase = smem_u32(smem);

  auto issue = [&](int kb) {
    if (kb < nkb) {
      const uint32_t dst = sbase + (kb & 1) * STAGE;
      for (int id = threadIdx.x; id < kLpKeys * (KD / 8); id += 128) {
        const int r = id / (KD / 8), c = id % (KD / 8) * 8;
        const int key = kb * kLpKeys + r;
        const bool valid = key >= klo && key < kmax && c < qd;
        const long long kr = valid ? kbase + key : 0;
        const bf16* src = c < dimp ? kv + kr * ld_kv + head * hw + c : lat + kr * ld_lat + rankp + (valid ? c - dimp : 0);
        cp_async16(dst + r * KP + c * 2, src, valid);
      }
      for (int id = threadIdx.x; id < kLpKeys * (VD / 8); id += 128) {
        const int r = id / (VD / 8), c = id % (VD / 8) * 8;
        const int key = kb * kLpKeys + r;
        const bool valid = key >= klo && key < kmax && c < vdimp;
        const long long kr = valid ? kbase + key : 0;
        cp_async16(dst + kLpKeys * KP + r * VP + c * 2, kv + kr * ld_kv + head * hw + dimp + (valid ? c : 0), valid);
      }
    }
    cp_async_commit();
  };
  issue(kb0);

  // rows R0 and R0 + 8 of this warp's tile are tokens t0, t1
  const int t0 = warp * 16 + g, t1 = t0 + 8;
  const bool v0 = t0 < ntok, v1 = t1 < ntok;
  const int qpos0 = pos0 + t0, qpos1 = pos0 + t1;
  uint32_t qa[KS][4];
  {
    const bf16* q0 = q + static_cast<long long>(row0 + t0) * ld_q + head * qd;
    const bf16* q1 = q + static_cast<long long>(row0 + t1) * ld_q + head * qd;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const int c = ks * 16 + 2 * tq;
      qa[ks][0] = v0 && c < qd ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
      qa[ks][1] = v1 && c < qd ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
      qa[ks][2] = v0 && c + 8 < qd ? *reinterpret_cast<const uint32_t*>(q0 + c + 8) : 0u;
      qa[ks][3] = v1 && c + 8 < qd ? *reinterpret_cast<const uint32_t*>(q1 + c + 8) : 0u;
    }
  }
  float o[NT][4];
#pragma unroll
  for (int x = 0; x < NT; ++x) o[x][0] = o[x][1] = o[x][2] = o[x][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  const int lm_mi = lane >> 3, lm_r = lane & 7;
  const int wlast = pos0 + min(ntok - 1, warp * 16 + 15);           // last query of the warp, first key of its first query
  const int wfirst = window > 0 ? pos0 + warp * 16 - window + 1 : 0;
  const int lo0 = window > 0 ? qpos0 - window + 1 : 0, lo1 = window > 0 ? qpos1 - window + 1 : 0;

  for (int kb = kb0; kb < nkb; ++kb) {
    issue(kb + 1);
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t kbuf = sbase + (kb & 1) * STAGE, vbuf = kbuf + kLpKeys * KP;
    const int key0 = kb * kLpKeys;
    if (key0 <= wlast && warp * 16 < ntok && key0 + kLpKeys > wfirst) {
      float s[8][4];
#pragma unroll
      for (int x = 0; x < 8; ++x) s[x][0] = s[x][1] = s[x][2] = s[x][3] = 0.f;
#pragma unroll
      for (int kg = 0; kg < 4; ++kg) {
        const uint32_t ka = kbuf + (kg * 16 + (lm_mi >> 1) * 8 + lm_r) * KP + (lm_mi & 1) * 16;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(ka + ks * 32, b0, b1, b2, b3);
          mma_bf16_16816(s[2 * kg], qa[ks], b0, b1);
          mma_bf16_16816(s[2 * kg + 1], qa[ks], b2, b3);
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        const int k0 = key0 + x * 8 + 2 * tq, k1 = k0 + 1;
        s[x][0] = v0 && k0 <= qpos0 && k0 >= lo0 ? s[x][0] * scale_log2 : -INFINITY;
        s[x][1] = v0 && k1 <= qpos0 && k1 >= lo0 ? s[x][1] * scale_log2 : -INFINITY;
        s[x][2] = v1 && k0 <= qpos1 && k0 >= lo1 ? s[x][2] * scale_log2 : -INFINITY;
        s[x][3] = v1 && k1 <= qpos1 && k1 >= lo1 ? s[x][3] * scale_log2 : -INFINITY;
        mx0 = fmaxf(mx0, fmaxf(s[x][0], s[x][1]));
        mx1 = fmaxf(mx1, fmaxf(s[x][2], s[x][3]));
      }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
      // a row with nothing visible yet keeps -inf: subtract 0 instead so that exp2 gives 0, not NaN
      const float sub0 = mn0 == -INFINITY ? 0.f : mn0, sub1 = mn1 == -INFINITY ? 0.f : mn1;
      const float corr0 = exp2f(m0 - sub0), corr1 = exp2f(m1 - sub1);
      float ls0 = 0.f, ls1 = 0.f;
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        s[x][0] = exp2f(s[x][0] - sub0); s[x][1] = exp2f(s[x][1] - sub0);
        s[x][2] = exp2f(s[x][2] - sub1); s[x][3] = exp2f(s[x][3] - sub1);
        ls0 += s[x][0] + s[x][1];
        ls1 += s[x][2] + s[x][3];
      }
      ls0 += __shfl_xor_sync(0xffffffffu, ls0, 1);
      ls0 += __shfl_xor_sync(0xffffffffu, ls0, 2);
      ls1 += __shfl_xor_sync(0xffffffffu, ls1, 1);
      ls1 += __shfl_xor_sync(0xffffffffu, ls1, 2);
      l0 = l0 * corr0 + ls0;
      l1 = l1 * corr1 + ls1;
      m0 = mn0;
      m1 = mn1;
#pragma unroll
      for (int x = 0; x < NT; ++x) { o[x][0] *= corr0; o[x][1] *= corr0; o[x][2] *= corr1; o[x][3] *= corr1; }
#pragma unroll
      for (int kg = 0; kg < 4; ++kg) {
        uint32_t ph[4], pl[4];
        split2(s[2 * kg][0], s[2 * kg][1], ph[0], pl[0]);
        split2(s[2 * kg][2], s[2 * kg][3], ph[1], pl[1]);
        split2(s[2 * kg + 1][0], s[2 * kg + 1][1], ph[2], pl[2]);
        split2(s[2 * kg + 1][2], s[2 * kg + 1][3], ph[3], pl[3]);
        const uint32_t va = vbuf + (kg * 16 + (lm_mi & 1) * 8 + lm_r) * VP + (lm_mi >> 1) * 16;
#pragma unroll
        for (int dp = 0; dp < NT / 2; ++dp) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(va + dp * 32, b0, b1, b2, b3);
          mma_bf16_16816(o[2 * dp], ph, b0, b1);
          mma_bf16_16816(o[2 * dp + 1], ph, b2, b3);
          mma_bf16_16816(o[2 * dp], pl, b0, b1);
          mma_bf16_16816(o[2 * dp + 1], pl, b2, b3);
        }
      }
    }
    __syncthreads();   // every warp is done with this stage before it is refilled
  }
  cp_async_wait<0>();
  float inv0 = l0 > 0.f ? 1.f / l0 : 0.f, inv1 = l1 > 0.f ? 1.f / l1 : 0.f;
  if (sink != nullptr) {
    const float sk = sink[head] * kLog2e;
    const float M0 = fmaxf(m0, sk), M1 = fmaxf(m1, sk), f0 = exp2f(m0 - M0), f1 = exp2f(m1 - M1);
    inv0 = f0 / (l0 * f0 + exp2f(sk - M0));
    inv1 = f1 / (l1 * f1 + exp2f(sk - M1));
  }
  if (gate != nullptr) {
    if (v0) inv0 *= 1.f / (1.f + expf(-__bfloat162float(gate[(row0 + t0) * ld_gate + head])));
    if (v1) inv1 *= 1.f / (1.f + expf(-__bfloat162float(gate[(row0 + t1) * ld_gate + head])));
  }
  bf16* o0 = out + static_cast<long long>(row0 + t0) * ld_out + head * vdimp;
  bf16* o1 = out + static_cast<long long>(row0 + t1) * ld_out + head * vdimp;
#pragma unroll
  for (int x = 0; x < NT; ++x) {
    const int col = x * 8 + 2 * tq;
    if (col >= vdimp) continue;
    if (v0) *reinterpret_cast<uint32_t*>(o0 + col) = pack_bf16(o[x][0] * inv0, o[x][1] * inv0);
    if (v1) *reinterpret_cast<uint32_t*>(o1 + col) = pack_bf16(o[x][2] * inv1, o[x][3] * inv1);
  }
}

template <int NT>
static int launch_latent(const void* q, const void* cache, const int* bt, int max_blocks, const int* bt_row, const int* rows,
                         const int* ctx_len, int block_size, int n, int heads, int rankp, int kd, int row, float scale, int window,
                         const float* sink, int splits, void* out, float* ws, int* status,
                         cudaStream_t stream) {
  static PerDeviceOnce configured;
  const int rc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(latent_attn_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLatMaxSmem));
  });
  if (rc != 0) return rc;
  const LatentSmem L = latent_smem(kd, row);
  const int smem = L.total, groups = heads > 16 ? (heads + 31) / 32 : 1;
  const long long at = static_cast<long long>(heads) * n, ctas = static_cast<long long>(groups) * n;
  if (L.stages < 2 || smem > kLatMaxSmem || ctas > 0x7fffffffll) return -11;
  float* part_lse = ws != nullptr ? ws + at * splits * rankp : nullptr;
  latent_attn_kernel<NT><<<dim3(static_cast<unsigned>(ctas), splits), kLatThreads, smem, stream>>>(
      static_cast<const bf16*>(q), static_cast<const bf16*>(cache), bt, max_blocks, bt_row, rows, ctx_len, block_size, n, heads,
      groups, rankp, kd, row, scale * kLog2e, window, sink, splits, static_cast<bf16*>(out), ws, part_lse,
      status);
  if (splits > 1)
    latent_merge_kernel<<<static_cast<unsigned>(at), 128, 0, stream>>>(ws, part_lse, splits, rankp, static_cast<bf16*>(out));
  return static_cast<int>(cudaGetLastError());
}

template <int KD, int VD>
static int launch_latent_prefill(const void* q, long long ld_q, const void* kv, long long ld_kv, const void* lat, long long ld_lat,
                                 const void* tiles, const int* base, int n_tiles, int heads, int dimp, int rotp, int rankp,
                                 int vdimp, float scale, int window, const float* sink, const void* gate, long long ld_gate,
                                 void* out, long long ld_out, cudaStream_t stream) {
  constexpr int smem = 2 * kLpKeys * (KD * 2 + VD * 2 + 32);
  static PerDeviceOnce configured;
  const int rc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(latent_prefill_kernel<KD, VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  });
  if (rc != 0) return rc;
  latent_prefill_kernel<KD, VD><<<dim3(n_tiles, heads), 128, smem, stream>>>(
      static_cast<const bf16*>(q), ld_q, static_cast<const bf16*>(kv), ld_kv, static_cast<const bf16*>(lat), ld_lat,
      static_cast<const int4*>(tiles), base, dimp, rotp, rankp, vdimp, scale * kLog2e, window, sink,
      static_cast<const bf16*>(gate), ld_gate, static_cast<bf16*>(out), ld_out);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace dmoe

using namespace dmoe;

extern "C" int dmoe_latent_prep(int is_f32, void* y, long long ld, const int* positions, const long long* slots, void* cache, int T,
                                int heads, int dim, int rot_dim, int rank, int row, int rot, int interleaved, const void* table,
                                int max_pos, const float* norm_w, float eps, const int* loose, int n_loose, void* xq, void* qa,
                                const void* gate, void* recs, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (heads < 1 || dim < 1 || rot_dim < 0 || rank < 1 || rot < 0 || rot % 2 != 0 || rot > rot_dim || (rot > 0 && table == nullptr)) return -10;
  const int align = is_f32 ? 4 : 8;
  if (row % align != 0 || row < pad8(rank) + pad8(rot_dim)) return -10;
  if (ld % align != 0 || (reinterpret_cast<uintptr_t>(y) & 15) != 0 || (loose == nullptr && n_loose < T)) return -10;
  if (gate != nullptr && n_loose > 0 && recs == nullptr) return -10;
  if (T == 0) return 0;
  const int dimp = pad8(dim), rotp = pad8(rot_dim), rankp = pad8(rank);
  const bool vec = interleaved && rot == rotp && rot > 0;
#define DMOE_PREP(T_, VEC_)                                                                                                  \
  latent_prep_kernel<T_, VEC_><<<T, 256, 0, stream>>>(                                                                       \
      static_cast<T_*>(y), ld, positions, slots, static_cast<T_*>(cache), heads, dimp, rotp, rank, rankp, row, rot,          \
      interleaved, static_cast<const float2*>(table), max_pos, norm_w, eps, loose, n_loose, static_cast<T_*>(xq),            \
      static_cast<T_*>(qa), static_cast<const T_*>(gate), static_cast<int4*>(recs))
  if (is_f32 && vec) DMOE_PREP(float, true);
  else if (is_f32) DMOE_PREP(float, false);
  else if (vec) DMOE_PREP(bf16, true);
  else DMOE_PREP(bf16, false);
#undef DMOE_PREP
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_latent_attention(const void* qa, const void* cache, const int* block_tables, int max_blocks, const int* bt_row,
                                     const int* rows, const int* ctx_len, int block_size, int n, int heads, int rankp, int kd, int row,
                                     float scale, int window, const float* sink, int splits, void* out, float* workspace,
                                     int* status, void* stream_) {
  if (heads < 1 || heads > 65535 || rankp < 8 || rankp % 8 != 0 || kd % 8 != 0 || kd < rankp || row < kd || rankp > 512 || kd > 640) return -10;
  if (row % 16 != 8 || block_size % kLatPiece != 0) return -10;
  if ((reinterpret_cast<uintptr_t>(qa) & 15) != 0 || (reinterpret_cast<uintptr_t>(cache) & 15) != 0) return -10;
  if (splits < 1 || splits > 65535 || (splits > 1 && workspace == nullptr)) return -10;
  if (n == 0) return 0;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
#define DMOE_LAT(NT_)                                                                                                   \
  return launch_latent<NT_>(qa, cache, block_tables, max_blocks, bt_row, rows, ctx_len, block_size, n, heads, rankp, kd, \
                            row, scale, window, sink, splits, out, workspace, status, stream)
  if (rankp <= 128) DMOE_LAT(2);
  if (rankp <= 256) DMOE_LAT(4);
  DMOE_LAT(8);
#undef DMOE_LAT
}

extern "C" int dmoe_latent_gather(const void* cache, const int* block_tables, int max_blocks, const void* keys, int n,
                                  int block_size, int row, void* out, void* stream) {
  if (row < 8 || row % 8 != 0 || block_size < 1) return -10;
  if (n == 0) return 0;
  latent_gather_kernel<<<(n + 7) / 8, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(cache), block_tables, max_blocks, static_cast<const int2*>(keys), n, block_size, row / 8,
      static_cast<uint4*>(out));
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_latent_prefill(const void* q, long long ld_q, const void* kv, long long ld_kv, const void* lat, long long ld_lat,
                                   const void* tiles, const int* base, int n_tiles, int heads, int dimp, int rotp, int rankp,
                                   int vdimp, float scale, int window, const float* sink, const void* gate, long long ld_gate,
                                   void* out, long long ld_out, void* stream_) {
  if (n_tiles == 0) return 0;
  if (n_tiles < 0 || heads < 1 || heads > 65535 || dimp % 8 != 0 || rotp % 8 != 0 || rankp % 8 != 0 || vdimp % 8 != 0) return -10;
  if (ld_q % 8 != 0 || ld_kv % 8 != 0 || ld_lat % 8 != 0 || ld_out % 8 != 0 || tiles == nullptr || base == nullptr) return -10;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  const int kd = dimp + rotp;
#define DMOE_LP(KD_, VD_)                                                                                               \
  if (kd <= KD_ && vdimp <= VD_)                                                                                        \
    return launch_latent_prefill<KD_, VD_>(q, ld_q, kv, ld_kv, lat, ld_lat, tiles, base, n_tiles, heads, dimp, rotp, rankp, \
                                           vdimp, scale, window, sink, gate, ld_gate, out, ld_out, stream)
  DMOE_LP(96, 64);
  DMOE_LP(128, 128);
  DMOE_LP(192, 128);
#undef DMOE_LP
  return -11;
}
