// Paged attention for sm_100a: one kernel serves decode tokens and prefill tokens.
//
// Every query token t attends to the first ctx_len[t] tokens of the paged KV cache of its sequence
// (block table row bt_row[t]); a decode token has ctx_len = sequence length, prompt token i of a prefill has
// ctx_len = i + 1 (causal), its K/V having been appended to the cache by rope_kv_append before this kernel runs.
// So mixed prefill + decode batches need no second code path.
//
// The work of one CTA is (token, kv head, kv split): the GQ query heads that share the kv head are processed
// together, so every K/V byte is read once per group. It is a bandwidth problem (256 B of K and of V per
// cached token and kv head), so the kernel is built around wide loads kept in flight rather than around
// CUDA-core FLOPs: K/V rows stream through per-warp cp.async rings in shared memory and the GQ x 16-token score and
// output tiles run on the tensor cores (mma.sync m16n8k16: the group is far too small for a tcgen05 tile); softmax is online (base 2); the 16 (warp, lane-group) partial states are merged through
// shared memory. With splits > 1 ("flash decoding") partial outputs + log-sum-exp go to a workspace and a
// second kernel merges them.
//
// Cache layout: K and V each [num_blocks, block_size, kv_heads, head_dim] bf16.
// Reference behaviour covered: vLLM paged attention / flash_attn_with_kvcache reached from
// disagmoe/models/attention.py:150-155,219 with metadata built at disagmoe/frontend/engine.py:429-485.
#include "dmoe_kernels.h"
#include "mma_sync.cuh"

namespace dmoe {

constexpr int kAttnThreads = 128;
constexpr int kAttnParts = 16;  // 4 warps x 4 lane groups

struct alignas(16) bf16x8a {
  __nv_bfloat162 v[4];
};

__device__ __forceinline__ void cvt8(const bf16x8a& p, float* f) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = __bfloat1622float2(p.v[i]);
    f[2 * i] = t.x;
    f[2 * i + 1] = t.y;
  }
}

// The decode kernel reads every K / V byte once per step: an evict-first L2 policy keeps that stream from pushing the
// small hot tensors of the neighbouring kernels (residual rows, norm and gate weights, staged activations) out of L2.
__device__ __forceinline__ uint64_t l2_stream_policy() {
  uint64_t p;
  asm volatile("createpolicy.fractional.L2::evict_first.b64 %0, 1.0;" : "=l"(p));
  return p;
}
__device__ __forceinline__ void cp_async16_stream(uint32_t dst, const void* src, bool valid, uint64_t policy) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global.L2::cache_hint [%0], [%1], 16, %2, %3;" ::"r"(dst), "l"(src), "r"(sz), "l"(policy)
               : "memory");
}
// Options of the EXT instantiations of both kernels (plain ones compile without them):
//   window > 0: a query at position p sees only keys in (p - window, p];
//   chunk > 0: it sees only keys of its own chunk of `chunk` positions, counted from position 0;
//   cap_log2 > 0: score <- cap * tanh(score / cap) before the softmax (cap_log2 = cap * log2 e, cap_in = 2 scale log2 e / cap);
//   sink != NULL: exp(sink[head]) enters the softmax denominator (no key, no value);
//   temp_every > 0: scores are multiplied by the query temperature 1 + temp_coef ln(floor((p + 1) / temp_every) + 1);
//   gate != NULL: head outputs are multiplied by sigmoid(gate[row, head]) (row stride ld_gate);
//   gq: query heads per kv head where the instantiation leaves it open (GQ = 0).
// The EXT kernels also keep the softmax weights at fp32 accuracy in the P V product: P = hi + lo, both bf16, two MMAs.
struct AttnExt {
  int window, chunk;
  float cap_in, cap_log2;
  const float* sink;
  int gq;
  const void* gate;
  long long ld_gate;
  float temp_coef;
  int temp_every;
};
__device__ __forceinline__ float query_temperature(const AttnExt& x, int p) {
  return x.temp_every > 0 ? 1.f + x.temp_coef * logf(static_cast<float>((p + 1) / x.temp_every + 1)) : 1.f;
}
template <typename T>
__device__ __forceinline__ float head_gate(const AttnExt& x, long long row, int head) {
  return x.gate != nullptr ? 1.f / (1.f + expf(-static_cast<float>(static_cast<const T*>(x.gate)[row * x.ld_gate + head]))) : 1.f;
}
constexpr float kLog2e = 1.4426950408889634f;
// first key that a query at position p sees
__device__ __forceinline__ int first_key(int p, int window, int chunk) {
  int lo = window > 0 ? max(0, p - window + 1) : 0;
  if (chunk > 0) lo = max(lo, p / chunk * chunk);
  return lo;
}
// 16-byte chunk c of tile row r in shared memory: rows of 128 bytes and more permute their chunks by groups of eight, rows of
// 64 bytes (two to a 128-byte line) by groups of four; either way eight rows of one column meet no bank twice.
template <int NCH>
__device__ __forceinline__ int swz(int c, int r) {
  static_assert(NCH == 4 || NCH % 8 == 0, "row size");
  return NCH == 4 ? c ^ ((r >> 1) & 3) : c ^ (r & 7);
}
// raw q.k -> score in base-2 units. tanh(x) = 1 - 2 / (exp(2x) + 1), good to ~1e-7 absolute.
template <bool EXT>
__device__ __forceinline__ float attn_score(float raw, float scale_log2, const AttnExt& x) {
  if (EXT && x.cap_log2 > 0.f) return x.cap_log2 * (1.f - __fdividef(2.f, exp2f(raw * x.cap_in) + 1.f));
  return raw * scale_log2;
}

constexpr int kAttnStages = 3;     // cp.async ring depth, per warp
constexpr int kAttnStageTok = 16;  // cached tokens per stage and warp (block_size must be a multiple of it)
constexpr int kAttnWarps = kAttnThreads / 32;

// Tensor-core formulation: the GQ query heads of one kv head are the (zero padded) 16 rows of an m16n8k16 tile.
// Each warp owns every 4th chunk of 16 cached tokens and streams them through its private cp.async ring
// (swizzled so that ldmatrix is bank-conflict free): S = Q K^T (2 n-tiles), online softmax on the accumulator
// fragments, P re-used in place as the A operand of O += P V (V read with ldmatrix.trans).
// VD: value size. GQ = 0: groups of ext.gq heads, at most 8 of which go to one CTA.
template <int HD, int VD, int GQ, bool EXT>
__global__ void __launch_bounds__(kAttnThreads)
paged_attn_kernel(const __nv_bfloat16* __restrict__ q, long long ld_q, const __nv_bfloat16* __restrict__ kcache,
                  const __nv_bfloat16* __restrict__ vcache, const int* __restrict__ block_tables, int max_blocks,
                  const int* __restrict__ bt_row, const int* __restrict__ ctx_len, int block_size, int n_kv,
                  float scale_log2, int splits, __nv_bfloat16* __restrict__ out, long long ld_out,
                  float* __restrict__ part_o, float* __restrict__ part_lse, AttnExt ext) {
  static_assert(GQ <= 8, "the query group must fit the first 8 rows of the MMA tile");
  constexpr int ROWB = HD * 2, ROWBV = VD * 2;       // bytes of one cached key / value row of one kv head
  constexpr int NCH = HD / 8, NCHV = VD / 8;         // 16-byte chunks per row
  constexpr int TILEB = kAttnStageTok * ROWB;        // K tile of one stage
  constexpr int STAGEB = TILEB + kAttnStageTok * ROWBV;
  constexpr int WARPB = kAttnStages * STAGEB;
  constexpr int CPL = kAttnStageTok * NCH / 32, CPLV = kAttnStageTok * NCHV / 32;   // 16-byte copies per lane per tile
  constexpr int KS = HD / 16;                        // k-steps of Q K^T
  constexpr int NT = VD / 8;                         // n-tiles of the output
  __shared__ float s_m[kAttnWarps][8];
  __shared__ float s_l[kAttnWarps][8];
  extern __shared__ __align__(128) uint8_t s_dyn[];  // per-warp rings; reused as [warps][heads][VD] floats at the end

  pdl_trigger();
  pdl_wait();      // q, the new K / V rows and the sequence tables come from the kernels before this one
  const int gq = GQ > 0 ? GQ : ext.gq, nsub = GQ > 0 ? 1 : (gq + 7) / 8;
  const int t = blockIdx.x, hkv = blockIdx.y / nsub, split = blockIdx.z;
  const int sub0 = (blockIdx.y % nsub) * 8;          // this CTA's heads of the group: sub0 .. sub0 + gn - 1
  const int gn = GQ > 0 ? GQ : min(8, gq - sub0), head0 = hkv * gq + sub0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tq = lane & 3;            // accumulator row / column-pair of this lane
  const int n_q = n_kv * gq;

  const int len = ctx_len[t];
  const int row = bt_row != nullptr ? bt_row[t] : t;
  const int* bt = block_tables + static_cast<long long>(row) * max_blocks;
  // first visible token, and its block: the blocks from there on are dealt out to the splits
  const int vis0 = EXT && len > 0 ? first_key(len - 1, ext.window, ext.chunk) : 0;
  const int blk0 = vis0 / block_size;
  const int nblk = (len + block_size - 1) / block_size - blk0;
  const int blk_per = (nblk + splits - 1) / splits;
  int c0 = min(len, (blk0 + split * blk_per) * block_size);
  const int c1 = min(len, (blk0 + (split + 1) * blk_per) * block_size);
  if (EXT) c0 = max(c0, vis0 / kAttnStageTok * kAttnStageTok);
  const int nchunk = (c1 - c0 + kAttnStageTok - 1) / kAttnStageTok;
  const int my_chunks = nchunk > warp ? (nchunk - warp + kAttnWarps - 1) / kAttnWarps : 0;
  const uint32_t ring = smem_u32(s_dyn) + warp * WARPB;
  const uint64_t stream_policy = l2_stream_policy();

  auto issue = [&](int j) {
    if (j < my_chunks) {
      const int tok0 = c0 + (warp + j * kAttnWarps) * kAttnStageTok;
      const long long blk = bt[tok0 / block_size];
      const long long slot0 = blk * block_size + tok0 % block_size;
      const uint32_t dst0 = ring + (j % kAttnStages) * STAGEB;
#pragma unroll
      for (int i = 0; i < CPL; ++i) {
        const int id = lane + i * 32;
        const int r = id / NCH, c = id % NCH;
        const bool valid = tok0 + r < c1;
        const long long off = valid ? ((slot0 + r) * n_kv + hkv) * HD + c * 8 : 0;
        cp_async16_stream(dst0 + r * ROWB + (swz<NCH>(c, r) << 4), kcache + off, valid, stream_policy);
        if (HD == VD) cp_async16_stream(dst0 + TILEB + r * ROWBV + (swz<NCHV>(c, r) << 4), vcache + off, valid, stream_policy);
      }
      if (HD != VD) {
#pragma unroll
        for (int i = 0; i < CPLV; ++i) {
          const int id = lane + i * 32;
          const int r = id / NCHV, c = id % NCHV;
          const bool valid = tok0 + r < c1;
          const long long off = valid ? ((slot0 + r) * n_kv + hkv) * VD + c * 8 : 0;
          cp_async16_stream(dst0 + TILEB + r * ROWBV + (swz<NCHV>(c, r) << 4), vcache + off, valid, stream_policy);
        }
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int j = 0; j < kAttnStages - 1; ++j) issue(j);

  // Q fragments (rows >= gn are zero)
  uint32_t qa[KS][4];
  {
    const __nv_bfloat16* qp = q + static_cast<long long>(t) * ld_q + (head0 + g) * HD;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      qa[ks][0] = g < gn ? *reinterpret_cast<const uint32_t*>(qp + ks * 16 + 2 * tq) : 0u;
      qa[ks][2] = g < gn ? *reinterpret_cast<const uint32_t*>(qp + ks * 16 + 8 + 2 * tq) : 0u;
      qa[ks][1] = 0u;
      qa[ks][3] = 0u;
    }
  }
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m = -INFINITY, l = 0.f;
  const float temp = EXT ? query_temperature(ext, len - 1) : 1.f;

  // ldmatrix lane roles
  const int lm_mi = lane >> 3, lm_r = lane & 7;
  for (int j = 0; j < my_chunks; ++j) {
    issue(j + kAttnStages - 1);
    cp_async_wait<kAttnStages - 1>();
    __syncwarp();
    const uint32_t kb = ring + (j % kAttnStages) * STAGEB;
    const uint32_t vb = kb + TILEB;
    const int tok0 = c0 + (warp + j * kAttnWarps) * kAttnStageTok;
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
    {
      const int r = (lm_mi >> 1) * 8 + lm_r;          // token row this lane addresses
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        const int c = 2 * ks + (lm_mi & 1);
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(kb + r * ROWB + (swz<NCH>(c, r) << 4), b0, b1, b2, b3);
        mma_bf16_16816(s0, qa[ks], b0, b1);
        mma_bf16_16816(s1, qa[ks], b2, b3);
      }
    }
    // row g: tokens tok0 + 2 tq + {0, 1} (s0) and tok0 + 8 + 2 tq + {0, 1} (s1)
    const int tk = tok0 + 2 * tq;
    auto seen = [&](int j) { return j < c1 && (!EXT || j >= vis0); };
    float p00 = seen(tk) ? attn_score<EXT>(s0[0] * temp, scale_log2, ext) : -INFINITY;
    float p01 = seen(tk + 1) ? attn_score<EXT>(s0[1] * temp, scale_log2, ext) : -INFINITY;
    float p10 = seen(tk + 8) ? attn_score<EXT>(s1[0] * temp, scale_log2, ext) : -INFINITY;
    float p11 = seen(tk + 9) ? attn_score<EXT>(s1[1] * temp, scale_log2, ext) : -INFINITY;
    float mx = fmaxf(fmaxf(p00, p01), fmaxf(p10, p11));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    const float mn = fmaxf(m, mx);                     // finite: every chunk holds a visible token
    const float corr = exp2f(m - mn);
    p00 = exp2f(p00 - mn); p01 = exp2f(p01 - mn); p10 = exp2f(p10 - mn); p11 = exp2f(p11 - mn);
    float ls = p00 + p01 + p10 + p11;
    ls += __shfl_xor_sync(0xffffffffu, ls, 1);
    ls += __shfl_xor_sync(0xffffffffu, ls, 2);
    l = l * corr + ls;
    m = mn;
#pragma unroll
    for (int i = 0; i < NT; ++i) { o[i][0] *= corr; o[i][1] *= corr; }
    uint32_t pa[4] = {pack_bf16(p00, p01), 0u, pack_bf16(p10, p11), 0u};
    const uint32_t pl[4] = {pack_bf16(bf16_rest(p00), bf16_rest(p01)), 0u, pack_bf16(bf16_rest(p10), bf16_rest(p11)), 0u};
    {
      const int r = (lm_mi & 1) * 8 + lm_r;
#pragma unroll
      for (int dp = 0; dp < NT / 2; ++dp) {
        const int c = 2 * dp + (lm_mi >> 1);
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(vb + r * ROWBV + (swz<NCHV>(c, r) << 4), b0, b1, b2, b3);
        mma_bf16_16816(o[2 * dp], pa, b0, b1);
        mma_bf16_16816(o[2 * dp + 1], pa, b2, b3);
        if (EXT) {
          mma_bf16_16816(o[2 * dp], pl, b0, b1);
          mma_bf16_16816(o[2 * dp + 1], pl, b2, b3);
        }
      }
    }
    __syncwarp();   // every lane is done with this ring slot before it is refilled
  }
  cp_async_wait<0>();
  __syncthreads();

  // merge the warps' partial states
  float* s_acc = reinterpret_cast<float*>(s_dyn);   // [warps][gn][VD]
  if (g < gn) {
    if (tq == 0) { s_m[warp][g] = m; s_l[warp][g] = l; }
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      s_acc[(warp * gn + g) * VD + i * 8 + 2 * tq] = o[i][0];
      s_acc[(warp * gn + g) * VD + i * 8 + 2 * tq + 1] = o[i][1];
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < gn * VD; idx += kAttnThreads) {
    const int gg = idx / VD, d = idx % VD;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < kAttnWarps; ++w) M = fmaxf(M, s_m[w][gg]);
    const int head = head0 + gg;
    const bool sunk = EXT && ext.sink != nullptr && split == 0;      // one split carries the sink
    const float sk = sunk ? ext.sink[head] * kLog2e : -INFINITY;
    M = fmaxf(M, sk);
    float L = sunk ? exp2f(sk - M) : 0.f, O = 0.f;
    if (M > -INFINITY) {
#pragma unroll
      for (int w = 0; w < kAttnWarps; ++w) {
        const float wgt = exp2f(s_m[w][gg] - M);
        L += s_l[w][gg] * wgt;
        O += s_acc[(w * gn + gg) * VD + d] * wgt;
      }
    }
    const float val = L > 0.f ? O / L : 0.f;
    if (splits == 1) {
      const float gated = EXT ? val * head_gate<__nv_bfloat16>(ext, t, head) : val;
      out[static_cast<long long>(t) * ld_out + head * VD + d] = __float2bfloat16(gated);
    } else {
      const long long pi = (static_cast<long long>(t) * n_q + head) * splits + split;
      part_o[pi * VD + d] = val;
      if (d == 0) part_lse[pi] = L > 0.f ? M + log2f(L) : -INFINITY;
    }
  }
}

// out[t, head] = sum_s softmax_s(lse) * part_o[t, head, s], gated
template <int VD>
__global__ void attn_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse, int splits,
                                  int n_q, __nv_bfloat16* __restrict__ out, long long ld_out, AttnExt ext) {
  const int t = blockIdx.x, head = blockIdx.y, d = threadIdx.x;
  const long long pi = (static_cast<long long>(t) * n_q + head) * splits;
  float M = -INFINITY;
  for (int s = 0; s < splits; ++s) M = fmaxf(M, part_lse[pi + s]);
  float L = 0.f, O = 0.f;
  if (M > -INFINITY) {
    for (int s = 0; s < splits; ++s) {
      const float w = exp2f(part_lse[pi + s] - M);
      L += w;
      O += w * part_o[(pi + s) * VD + d];
    }
  }
  out[static_cast<long long>(t) * ld_out + head * VD + d] =
      __float2bfloat16(L > 0.f ? O / L * head_gate<__nv_bfloat16>(ext, t, head) : 0.f);
}

// ---------------------------------------------------------------------------------------------------------------
// Tiled causal attention for prompt tokens (prefill, whole prompts or chunks of them).
//
// The per-token kernel above streams a prompt row's whole prefix for every row: O(n^2) K/V bytes per prompt with no
// reuse. Here a CTA owns a tile of 64 query rows = (64 / GQ consecutive prompt tokens) x (the GQ query heads of one kv
// head) and streams the sequence's K/V pages ONCE for the tile, 64 keys at a time, through a double-buffered
// cp.async ring shared by its four warps; each warp holds 16 query rows as mma.sync A fragments, computes S = Q K^T
// for the 64 keys, applies the causal mask (key position <= query position; the chunk's own K/V are already in the
// cache), runs the online softmax on the accumulator fragments and reuses P in registers as the A operand of O += P V.
// A chunk that continues a prompt attends to the cached prefix and to itself, so chunked prefill needs nothing else.
//
// tiles: one int4 per CTA column = {first row of the tile in q / out, tokens in the tile (<= 64 / GQ), block-table
// row of the sequence, position of the tile's first token}.
constexpr int kPreKeys = 64;       // keys per pipeline stage
constexpr int kPreRows = 64;       // query rows per CTA (4 warps x 16)

// 1 / denominator of a row with running maximum m (base 2) and sum l, the sink included; 0 for a row that saw nothing.
__device__ __forceinline__ float sink_inverse(float m, float l, float sink) {
  const float sk = sink * kLog2e, M = fmaxf(m, sk), f = exp2f(m - M);
  return f / (l * f + exp2f(sk - M));
}

template <int HD, int VD, int GQ, bool EXT>
__global__ void __launch_bounds__(128)
prefill_attn_kernel(const __nv_bfloat16* __restrict__ q, long long ld_q, const __nv_bfloat16* __restrict__ kcache,
                    const __nv_bfloat16* __restrict__ vcache, const int* __restrict__ block_tables, int max_blocks,
                    const int4* __restrict__ tiles, int block_size, int n_kv, float scale_log2,
                    __nv_bfloat16* __restrict__ out, long long ld_out, AttnExt ext) {
  constexpr int ROWB = HD * 2, ROWBV = VD * 2;
  constexpr int NCH = HD / 8, NCHV = VD / 8;        // 16-byte chunks per K / V row
  constexpr int TILEB = kPreKeys * ROWB;
  constexpr int STAGEB = TILEB + kPreKeys * ROWBV;  // K tile then V tile
  constexpr int CPT = kPreKeys * NCH / 128, CPTV = kPreKeys * NCHV / 128;   // 16-byte copies per thread per tile
  constexpr int KS = HD / 16;                       // k-steps of Q K^T
  constexpr int NT = VD / 8;                        // n-tiles of the output
  extern __shared__ __align__(128) uint8_t s_pre[];

  const int4 tile = tiles[blockIdx.x];
  const int row0 = tile.x, ntok = tile.y, pos0 = tile.w;
  const int hkv = blockIdx.y, gq = GQ > 0 ? GQ : ext.gq;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tq = lane & 3;
  const int* bt = block_tables + static_cast<long long>(tile.z) * max_blocks;
  const int kmax = pos0 + ntok;                     // keys [0, kmax) exist for the last token of the tile
  const int nkb = (kmax + kPreKeys - 1) / kPreKeys;
  const int kb0 = EXT ? first_key(pos0, ext.window, ext.chunk) / kPreKeys : 0;   // first block anyone sees
  const uint32_t sbase = smem_u32(s_pre);

  auto issue = [&](int kb) {
    if (kb < nkb) {
      const uint32_t dst0 = sbase + (kb & 1) * STAGEB;
#pragma unroll
      for (int i = 0; i < CPT; ++i) {
        const int id = threadIdx.x + i * 128;
        const int r = id / NCH, c = id % NCH;
        const int key = kb * kPreKeys + r;
        const bool valid = key < kmax;
        long long off = 0;
        if (valid) {
          const long long blk = bt[key / block_size];
          off = ((blk * block_size + key % block_size) * n_kv + hkv) * HD + c * 8;
        }
        cp_async16(dst0 + r * ROWB + (swz<NCH>(c, r) << 4), kcache + off, valid);
        if (HD == VD) cp_async16(dst0 + TILEB + r * ROWBV + (swz<NCHV>(c, r) << 4), vcache + off, valid);
      }
      if (HD != VD) {
#pragma unroll
        for (int i = 0; i < CPTV; ++i) {
          const int id = threadIdx.x + i * 128;
          const int r = id / NCHV, c = id % NCHV;
          const int key = kb * kPreKeys + r;
          const bool valid = key < kmax;
          long long off = 0;
          if (valid) {
            const long long blk = bt[key / block_size];
            off = ((blk * block_size + key % block_size) * n_kv + hkv) * VD + c * 8;
          }
          cp_async16(dst0 + TILEB + r * ROWBV + (swz<NCHV>(c, r) << 4), vcache + off, valid);
        }
      }
    }
    cp_async_commit();
  };
  issue(kb0);

  // Q fragments: this warp's rows R0 = warp * 16 + g and R0 + 8; row R = (token R / gq, head R % gq)
  const int R0 = warp * 16 + g, R1 = R0 + 8;
  const int t0 = R0 / gq, t1 = R1 / gq;
  const int head0 = hkv * gq + R0 % gq, head1 = hkv * gq + R1 % gq;
  const bool v0 = t0 < ntok, v1 = t1 < ntok;
  const int qpos0 = pos0 + t0, qpos1 = pos0 + t1;
  uint32_t qa[KS][4];
  {
    const __nv_bfloat16* q0 = q + static_cast<long long>(row0 + t0) * ld_q + head0 * HD;
    const __nv_bfloat16* q1 = q + static_cast<long long>(row0 + t1) * ld_q + head1 * HD;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      qa[ks][0] = v0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 2 * tq) : 0u;
      qa[ks][1] = v1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 2 * tq) : 0u;
      qa[ks][2] = v0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 8 + 2 * tq) : 0u;
      qa[ks][3] = v1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 8 + 2 * tq) : 0u;
    }
  }
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  const int lm_mi = lane >> 3, lm_r = lane & 7;
  // the warp's last query position: key blocks entirely behind it are skipped by this warp (causal)
  const int wlast = pos0 + min(ntok - 1, (warp * 16 + 15) / gq);
  // and, with a window or chunks, those entirely before the reach of its first query; a row's first visible key
  const int wfirst = EXT ? first_key(pos0 + warp * 16 / gq, ext.window, ext.chunk) : 0;
  const float temp0 = EXT ? query_temperature(ext, qpos0) : 1.f, temp1 = EXT ? query_temperature(ext, qpos1) : 1.f;
  const int lo0 = EXT ? first_key(qpos0, ext.window, ext.chunk) : 0;
  const int lo1 = EXT ? first_key(qpos1, ext.window, ext.chunk) : 0;

  for (int kb = kb0; kb < nkb; ++kb) {
    issue(kb + 1);
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t kbuf = sbase + (kb & 1) * STAGEB;
    const uint32_t vbuf = kbuf + TILEB;
    const int key0 = kb * kPreKeys;
    if (key0 <= wlast && warp * 16 / gq < ntok && (!EXT || key0 + kPreKeys > wfirst)) {
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
#pragma unroll
      for (int kg = 0; kg < 4; ++kg) {
        const int r = kg * 16 + (lm_mi >> 1) * 8 + lm_r;       // key row this lane addresses
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
          const int c = 2 * ks + (lm_mi & 1);
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(kbuf + r * ROWB + (swz<NCH>(c, r) << 4), b0, b1, b2, b3);
          mma_bf16_16816(s[2 * kg], qa[ks], b0, b1);
          mma_bf16_16816(s[2 * kg + 1], qa[ks], b2, b3);
        }
      }
      // mask + online softmax. s[nt][0..1]: row R0, keys key0 + nt * 8 + 2 tq + {0, 1}; s[nt][2..3]: row R1
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const int k0 = key0 + nt * 8 + 2 * tq;
        const bool a0 = v0 && k0 <= qpos0 && (!EXT || k0 >= lo0), a1 = v0 && k0 + 1 <= qpos0 && (!EXT || k0 + 1 >= lo0);
        const bool b0 = v1 && k0 <= qpos1 && (!EXT || k0 >= lo1), b1 = v1 && k0 + 1 <= qpos1 && (!EXT || k0 + 1 >= lo1);
        s[nt][0] = a0 ? attn_score<EXT>(s[nt][0] * temp0, scale_log2, ext) : -INFINITY;
        s[nt][1] = a1 ? attn_score<EXT>(s[nt][1] * temp0, scale_log2, ext) : -INFINITY;
        s[nt][2] = b0 ? attn_score<EXT>(s[nt][2] * temp1, scale_log2, ext) : -INFINITY;
        s[nt][3] = b1 ? attn_score<EXT>(s[nt][3] * temp1, scale_log2, ext) : -INFINITY;
        mx0 = fmaxf(mx0, fmaxf(s[nt][0], s[nt][1]));
        mx1 = fmaxf(mx1, fmaxf(s[nt][2], s[nt][3]));
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
      for (int nt = 0; nt < 8; ++nt) {
        s[nt][0] = exp2f(s[nt][0] - sub0); s[nt][1] = exp2f(s[nt][1] - sub0);
        s[nt][2] = exp2f(s[nt][2] - sub1); s[nt][3] = exp2f(s[nt][3] - sub1);
        ls0 += s[nt][0] + s[nt][1];
        ls1 += s[nt][2] + s[nt][3];
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
      for (int i = 0; i < NT; ++i) { o[i][0] *= corr0; o[i][1] *= corr0; o[i][2] *= corr1; o[i][3] *= corr1; }
      // O += P V, 16 keys per k-step: P re-used in place as the A operand
#pragma unroll
      for (int kg = 0; kg < 4; ++kg) {
        const uint32_t pa[4] = {pack_bf16(s[2 * kg][0], s[2 * kg][1]), pack_bf16(s[2 * kg][2], s[2 * kg][3]),
                                pack_bf16(s[2 * kg + 1][0], s[2 * kg + 1][1]), pack_bf16(s[2 * kg + 1][2], s[2 * kg + 1][3])};
        uint32_t pl[4] = {0u, 0u, 0u, 0u};
        if (EXT) {
          pl[0] = pack_bf16(bf16_rest(s[2 * kg][0]), bf16_rest(s[2 * kg][1]));
          pl[1] = pack_bf16(bf16_rest(s[2 * kg][2]), bf16_rest(s[2 * kg][3]));
          pl[2] = pack_bf16(bf16_rest(s[2 * kg + 1][0]), bf16_rest(s[2 * kg + 1][1]));
          pl[3] = pack_bf16(bf16_rest(s[2 * kg + 1][2]), bf16_rest(s[2 * kg + 1][3]));
        }
        const int r = kg * 16 + (lm_mi & 1) * 8 + lm_r;
#pragma unroll
        for (int dp = 0; dp < NT / 2; ++dp) {
          const int c = 2 * dp + (lm_mi >> 1);
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(vbuf + r * ROWBV + (swz<NCHV>(c, r) << 4), b0, b1, b2, b3);
          mma_bf16_16816(o[2 * dp], pa, b0, b1);
          mma_bf16_16816(o[2 * dp + 1], pa, b2, b3);
          if (EXT) {
            mma_bf16_16816(o[2 * dp], pl, b0, b1);
            mma_bf16_16816(o[2 * dp + 1], pl, b2, b3);
          }
        }
      }
    }
    __syncthreads();   // every warp is done with this stage before it is refilled
  }
  cp_async_wait<0>();

  float inv0 = l0 > 0.f ? 1.f / l0 : 0.f, inv1 = l1 > 0.f ? 1.f / l1 : 0.f;
  if (EXT && ext.sink != nullptr) {
    inv0 = sink_inverse(m0, l0, ext.sink[head0]);
    inv1 = sink_inverse(m1, l1, ext.sink[head1]);
  }
  if (EXT && ext.gate != nullptr) {
    if (v0) inv0 *= head_gate<__nv_bfloat16>(ext, row0 + t0, head0);
    if (v1) inv1 *= head_gate<__nv_bfloat16>(ext, row0 + t1, head1);
  }
  if (v0) {
    __nv_bfloat16* op = out + static_cast<long long>(row0 + t0) * ld_out + head0 * VD;
#pragma unroll
    for (int i = 0; i < NT; ++i)
      *reinterpret_cast<uint32_t*>(op + i * 8 + 2 * tq) = pack_bf16(o[i][0] * inv0, o[i][1] * inv0);
  }
  if (v1) {
    __nv_bfloat16* op = out + static_cast<long long>(row0 + t1) * ld_out + head1 * VD;
#pragma unroll
    for (int i = 0; i < NT; ++i)
      *reinterpret_cast<uint32_t*>(op + i * 8 + 2 * tq) = pack_bf16(o[i][2] * inv1, o[i][3] * inv1);
  }
}

// Options of a launch as the kernels take them (softcap <= 0: none; window, chunk <= 0: every key).
static AttnExt make_ext(float scale, int window, int chunk, float softcap, const float* sink, int gq, const DmoeAttnExtra* extra) {
  AttnExt x;
  x.gate = extra != nullptr ? extra->gate : nullptr;
  x.ld_gate = extra != nullptr ? extra->ld_gate : 0;
  x.temp_coef = extra != nullptr ? extra->temp_coef : 0.f;
  x.temp_every = extra != nullptr ? extra->temp_every : 0;
  x.sink = sink;
  x.gq = gq;
  x.window = window > 0 ? window : 0;
  x.chunk = chunk > 0 ? chunk : 0;
  x.cap_in = softcap > 0.f ? 2.f * scale * 1.4426950408889634f / softcap : 0.f;
  x.cap_log2 = softcap > 0.f ? softcap * 1.4426950408889634f : 0.f;
  return x;
}

template <int HD, int VD, int GQ, bool EXT>
static int launch_prefill(const void* q, long long ld_q, const void* kc, const void* vc, const int* bt, int max_blocks,
                          const void* tiles, int n_tiles, int block_size, int n_kv, float scale, void* out,
                          long long ld_out, AttnExt ext, cudaStream_t stream) {
  const size_t smem = 2 * static_cast<size_t>(kPreKeys) * (HD + VD) * 2;
  static PerDeviceOnce configured;
  const int crc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(prefill_attn_kernel<HD, VD, GQ, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 96 * 1024));
  });
  if (crc != 0) return crc;
  dim3 grid(n_tiles, n_kv);
  prefill_attn_kernel<HD, VD, GQ, EXT><<<grid, 128, smem, stream>>>(
      static_cast<const __nv_bfloat16*>(q), ld_q, static_cast<const __nv_bfloat16*>(kc),
      static_cast<const __nv_bfloat16*>(vc), bt, max_blocks, static_cast<const int4*>(tiles), block_size, n_kv,
      scale * 1.4426950408889634f, static_cast<__nv_bfloat16*>(out), ld_out, ext);
  return static_cast<int>(cudaGetLastError());
}

template <int HD, int VD, int GQ, bool EXT>
static int launch_attn(const void* q, long long ld_q, const void* kc, const void* vc, const int* bt, int max_blocks,
                       const int* bt_row, const int* ctx_len, int block_size, int T, int n_kv, float scale, int splits,
                       void* out, long long ld_out, float* part_o, float* part_lse, AttnExt ext, cudaStream_t stream) {
  const int gq = GQ > 0 ? GQ : ext.gq, nsub = (gq + 7) / 8;
  const size_t merge_b = static_cast<size_t>(kAttnWarps) * (gq < 8 ? gq : 8) * VD * sizeof(float);
  const size_t ring_b = static_cast<size_t>(kAttnWarps) * kAttnStages * kAttnStageTok * (HD + VD) * 2;
  const size_t smem = merge_b > ring_b ? merge_b : ring_b;
  static PerDeviceOnce configured;
  const int crc = configured.run([] {
    return static_cast<int>(cudaFuncSetAttribute(paged_attn_kernel<HD, VD, GQ, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 160 * 1024));
  });
  if (crc != 0) return crc;
  dim3 grid(T, n_kv * nsub, splits);
  cudaError_t e = launch_kernel(paged_attn_kernel<HD, VD, GQ, EXT>, grid, dim3(kAttnThreads), smem, stream,
      static_cast<const __nv_bfloat16*>(q), ld_q, static_cast<const __nv_bfloat16*>(kc),
      static_cast<const __nv_bfloat16*>(vc), bt, max_blocks, bt_row, ctx_len, block_size, n_kv,
      scale * 1.4426950408889634f, splits, static_cast<__nv_bfloat16*>(out), ld_out, part_o, part_lse, ext);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (splits > 1) {
    dim3 g2(T, n_kv * gq);
    attn_merge_kernel<VD><<<g2, VD, 0, stream>>>(part_o, part_lse, splits, n_kv * gq,
                                                  static_cast<__nv_bfloat16*>(out), ld_out, ext);
    e = cudaGetLastError();
  }
  return static_cast<int>(e);
}

}  // namespace dmoe

using namespace dmoe;

extern "C" long long dmoe_paged_attention_workspace_floats(int T, int n_q, int hd, int splits) {
  if (splits <= 1) return 0;
  return static_cast<long long>(T) * n_q * splits * (hd + 1);
}

// Instantiations: without options by head size and query group, with options by key and value size; -11: no tensor-core
// kernel for this shape.
template <bool EXT>
static int attn_dispatch(const void* q, long long ld_q, const void* kcache, const void* vcache, const int* block_tables,
                         int max_blocks, const int* bt_row, const int* ctx_len, int block_size, int T, int n_q, int n_kv,
                         int hd, int vd, float scale, int splits, void* out, long long ld_out, float* workspace, AttnExt ext,
                         cudaStream_t stream) {
  if (T == 0) return 0;
  if (n_kv < 1 || n_q % n_kv != 0 || splits < 1 || splits > 65535 || n_q > 65535 || block_size % kAttnStageTok != 0) return -10;
  if (splits > 1 && workspace == nullptr) return -12;
  const int gq = n_q / n_kv;
  float* part_o = workspace;
  float* part_lse = workspace != nullptr ? workspace + static_cast<long long>(T) * n_q * splits * vd : nullptr;
#define DMOE_ATTN(HD_, VD_, GQ_)                                                                                             \
  return launch_attn<HD_, VD_, GQ_, EXT>(q, ld_q, kcache, vcache, block_tables, max_blocks, bt_row, ctx_len, block_size, T, \
                                         n_kv, scale, splits, out, ld_out, part_o, part_lse, ext, stream)
  if constexpr (EXT) {
    if (gq > 64) return -11;
    if (hd == 128 && vd == 128) DMOE_ATTN(128, 128, 0);
    if (hd == 128 && vd == 64) DMOE_ATTN(128, 64, 0);
    if (hd == 64 && vd == 128) DMOE_ATTN(64, 128, 0);
    if (hd == 64 && vd == 64) DMOE_ATTN(64, 64, 0);
    if (hd == 64 && vd == 32) DMOE_ATTN(64, 32, 0);
  } else if (hd == 128) {
    switch (gq) {
      case 1: DMOE_ATTN(128, 128, 1);
      case 2: DMOE_ATTN(128, 128, 2);
      case 4: DMOE_ATTN(128, 128, 4);
      case 8: DMOE_ATTN(128, 128, 8);
    }
  } else if (hd == 64) {
    switch (gq) {
      case 1: DMOE_ATTN(64, 64, 1);
      case 2: DMOE_ATTN(64, 64, 2);
      case 4: DMOE_ATTN(64, 64, 4);
      case 8: DMOE_ATTN(64, 64, 8);
    }
  }
#undef DMOE_ATTN
  return -11;
}

extern "C" int dmoe_paged_attention(const void* q, long long ld_q, const void* kcache, const void* vcache,
                                    const int* block_tables, int max_blocks, const int* bt_row, const int* ctx_len,
                                    int block_size, int T, int n_q, int n_kv, int hd, float scale, int splits, void* out,
                                    long long ld_out, float* workspace, void* stream_) {
  return attn_dispatch<false>(q, ld_q, kcache, vcache, block_tables, max_blocks, bt_row, ctx_len, block_size, T, n_q, n_kv,
                              hd, hd, scale, splits, out, ld_out, workspace, make_ext(scale, 0, 0, 0.f, nullptr, 0, nullptr),
                              static_cast<cudaStream_t>(stream_));
}

// The same with a sliding window, chunks of positions that see no other chunk (0 = without), a score soft cap (0 = without) and a sink per head (NULL = without), value heads of another
// size than key heads, and query groups of up to 64 heads.
extern "C" int dmoe_paged_attention_ext(const void* q, long long ld_q, const void* kcache, const void* vcache,
                                        const int* block_tables, int max_blocks, const int* bt_row, const int* ctx_len,
                                        int block_size, int T, int n_q, int n_kv, int hd, int vd, float scale, int window,
                                        int chunk, float softcap, const float* sink, int splits, void* out, long long ld_out,
                                        float* workspace, const DmoeAttnExtra* extra, void* stream_) {
  if (n_kv < 1) return -10;
  return attn_dispatch<true>(q, ld_q, kcache, vcache, block_tables, max_blocks, bt_row, ctx_len, block_size, T, n_q, n_kv,
                             hd, vd, scale, splits, out, ld_out, workspace, make_ext(scale, window, chunk, softcap, sink, n_q / n_kv, extra),
                             static_cast<cudaStream_t>(stream_));
}

// Tokens per tile of dmoe_prefill_attention for a query group of n_q / n_kv heads.
extern "C" int dmoe_prefill_tile_tokens(int n_q, int n_kv) {
  if (n_kv < 1 || n_q % n_kv != 0) return 0;
  return kPreRows / (n_q / n_kv);
}

template <bool EXT>
static int prefill_dispatch(const void* q, long long ld_q, const void* kcache, const void* vcache, const int* block_tables,
                            int max_blocks, const void* tiles, int n_tiles, int block_size, int n_q, int n_kv, int hd, int vd,
                            float scale, void* out, long long ld_out, AttnExt ext, cudaStream_t stream) {
  if (n_tiles == 0) return 0;
  if (n_kv < 1 || n_q % n_kv != 0 || n_kv > 65535 || n_tiles < 0 || block_size < 1 || tiles == nullptr) return -10;
  const int gq = n_q / n_kv;
#define DMOE_PRE(HD_, VD_, GQ_)                                                                                          \
  return launch_prefill<HD_, VD_, GQ_, EXT>(q, ld_q, kcache, vcache, block_tables, max_blocks, tiles, n_tiles, block_size, \
                                            n_kv, scale, out, ld_out, ext, stream)
  if constexpr (EXT) {
    if (gq > kPreRows) return -11;
    if (hd == 128 && vd == 128) DMOE_PRE(128, 128, 0);
    if (hd == 128 && vd == 64) DMOE_PRE(128, 64, 0);
    if (hd == 64 && vd == 128) DMOE_PRE(64, 128, 0);
    if (hd == 64 && vd == 64) DMOE_PRE(64, 64, 0);
    if (hd == 64 && vd == 32) DMOE_PRE(64, 32, 0);
  } else if (hd == 128) {
    switch (gq) {
      case 1: DMOE_PRE(128, 128, 1);
      case 2: DMOE_PRE(128, 128, 2);
      case 4: DMOE_PRE(128, 128, 4);
      case 8: DMOE_PRE(128, 128, 8);
    }
  } else if (hd == 64) {
    switch (gq) {
      case 1: DMOE_PRE(64, 64, 1);
      case 2: DMOE_PRE(64, 64, 2);
      case 4: DMOE_PRE(64, 64, 4);
      case 8: DMOE_PRE(64, 64, 8);
    }
  }
#undef DMOE_PRE
  return -11;
}

extern "C" int dmoe_prefill_attention(const void* q, long long ld_q, const void* kcache, const void* vcache,
                                      const int* block_tables, int max_blocks, const void* tiles, int n_tiles,
                                      int block_size, int n_q, int n_kv, int hd, float scale, void* out, long long ld_out,
                                      void* stream_) {
  return prefill_dispatch<false>(q, ld_q, kcache, vcache, block_tables, max_blocks, tiles, n_tiles, block_size, n_q, n_kv,
                                 hd, hd, scale, out, ld_out, make_ext(scale, 0, 0, 0.f, nullptr, 0, nullptr),
                                 static_cast<cudaStream_t>(stream_));
}

extern "C" int dmoe_prefill_attention_ext(const void* q, long long ld_q, const void* kcache, const void* vcache,
                                          const int* block_tables, int max_blocks, const void* tiles, int n_tiles,
                                          int block_size, int n_q, int n_kv, int hd, int vd, float scale, int window,
                                          int chunk, float softcap, const float* sink, void* out, long long ld_out,
                                          const DmoeAttnExtra* extra, void* stream_) {
  if (n_kv < 1) return -10;
  return prefill_dispatch<true>(q, ld_q, kcache, vcache, block_tables, max_blocks, tiles, n_tiles, block_size, n_q, n_kv,
                                hd, vd, scale, out, ld_out, make_ext(scale, window, chunk, softcap, sink, n_q / n_kv, extra),
                                static_cast<cudaStream_t>(stream_));
}

// ---------------------------------------------------------------------------------------------------------------
// Attention of any shape in fp32 arithmetic on the CUDA cores (key size, value size and query group free; bf16 or fp32
// cache): the fp32 configuration, and head shapes without a tensor-core kernel. One CTA per (token, query head) walks
// the visible keys 128 at a time: one score per thread, online softmax, then one value column per thread.
namespace dmoe {

constexpr int kAnyKeys = 128;

template <typename T>
__global__ void __launch_bounds__(kAnyKeys)
any_attn_kernel(const T* __restrict__ q, long long q_head, long long q_row, const T* __restrict__ kcache, long long k_tok,
                const T* __restrict__ vcache, long long v_tok, const int* __restrict__ block_tables, int max_blocks,
                const int* __restrict__ bt_row, const int* __restrict__ rows, const int* __restrict__ ctx_len, int block_size,
                int n_q, int n_kv, int dk, int dv, float scale, int window, int chunk, float softcap, const float* __restrict__ sink,
                T* __restrict__ out, long long o_head, long long o_row, AttnExt ext) {
  extern __shared__ float s_any[];          // q [dk] | acc [dv]
  __shared__ float s_p[kAnyKeys];
  __shared__ long long s_slot[kAnyKeys];
  __shared__ float s_red[2][kAnyKeys / 32];
  float* s_q = s_any;
  float* s_acc = s_any + dk;
  const int head = blockIdx.y, tid = threadIdx.x;
  const int t = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;      // batch row whose context the query has
  const T* qp = q + blockIdx.x * q_row + head * q_head;
  const int hkv = head / (n_q / n_kv);
  const int len = ctx_len[t];
  const int* bt = block_tables + static_cast<long long>(bt_row != nullptr ? bt_row[t] : t) * max_blocks;
  for (int d = tid; d < dk; d += kAnyKeys) s_q[d] = static_cast<float>(qp[d]);
  for (int d = tid; d < dv; d += kAnyKeys) s_acc[d] = 0.f;
  __syncthreads();
  float m = -INFINITY, l = 0.f;
  scale *= query_temperature(ext, len - 1);
  for (int j0 = len > 0 ? first_key(len - 1, window, chunk) : 0; j0 < len; j0 += kAnyKeys) {
    const int n = min(kAnyKeys, len - j0);
    float s = -INFINITY;
    if (tid < n) {
      const int j = j0 + tid;
      const long long slot = static_cast<long long>(bt[j / block_size]) * block_size + j % block_size;
      const T* kr = kcache + slot * k_tok + hkv * dk;
      float acc = 0.f;
      for (int d = 0; d < dk; ++d) acc += s_q[d] * static_cast<float>(kr[d]);
      s = acc * scale;
      if (softcap > 0.f) s = softcap * tanhf(s / softcap);
      s_slot[tid] = slot;
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if ((tid & 31) == 0) s_red[0][tid >> 5] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(s_red[0][0], s_red[0][1]), fmaxf(s_red[0][2], s_red[0][3]));
    const float mn = fmaxf(m, mx);           // finite: a tile has at least one key
    const float p = tid < n ? expf(s - mn) : 0.f;
    s_p[tid] = p;
    float ps = p;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
    if ((tid & 31) == 0) s_red[1][tid >> 5] = ps;
    __syncthreads();
    const float corr = expf(m - mn);
    l = l * corr + (s_red[1][0] + s_red[1][1] + s_red[1][2] + s_red[1][3]);
    m = mn;
    for (int d = tid; d < dv; d += kAnyKeys) {
      float acc = s_acc[d] * corr;
      for (int j = 0; j < n; ++j) acc += s_p[j] * static_cast<float>(vcache[s_slot[j] * v_tok + hkv * dv + d]);
      s_acc[d] = acc;
    }
    __syncthreads();
  }
  float f = head_gate<T>(ext, t, head);
  if (sink != nullptr && len > 0) {
    const float mn = fmaxf(m, sink[head]);
    const float shrink = expf(m - mn);
    f *= shrink;
    l = l * shrink + expf(sink[head] - mn);
  }
  for (int d = tid; d < dv; d += kAnyKeys)
    out[blockIdx.x * o_row + head * o_head + d] = static_cast<T>(l > 0.f ? s_acc[d] * f / l : 0.f);
}

}  // namespace dmoe

extern "C" int dmoe_any_attention(int is_f32, const void* q, long long q_head, long long q_row, const void* kcache,
                                  long long k_tok, const void* vcache, long long v_tok, const int* block_tables, int max_blocks,
                                  const int* bt_row, const int* rows, const int* ctx_len, int block_size, int T, int n_q,
                                  int n_kv, int dk, int dv, float scale, int window, int chunk, float softcap, const float* sink, void* out,
                                  long long o_head, long long o_row, const DmoeAttnExtra* extra, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (T == 0) return 0;
  if (n_kv < 1 || n_q % n_kv != 0 || n_q > 65535 || block_size < 1 || dk < 1 || dv < 1 || dk + dv > 8192) return -10;
  const dim3 grid(T, n_q);
  const AttnExt ext = make_ext(scale, window, chunk, softcap, sink, n_q / n_kv, extra);
  const size_t smem = static_cast<size_t>(dk + dv) * sizeof(float);
  if (is_f32)
    any_attn_kernel<float><<<grid, kAnyKeys, smem, stream>>>(
        static_cast<const float*>(q), q_head, q_row, static_cast<const float*>(kcache), k_tok, static_cast<const float*>(vcache),
        v_tok, block_tables, max_blocks, bt_row, rows, ctx_len, block_size, n_q, n_kv, dk, dv, scale, window, chunk, softcap, sink,
        static_cast<float*>(out), o_head, o_row, ext);
  else
    any_attn_kernel<__nv_bfloat16><<<grid, kAnyKeys, smem, stream>>>(
        static_cast<const __nv_bfloat16*>(q), q_head, q_row, static_cast<const __nv_bfloat16*>(kcache), k_tok,
        static_cast<const __nv_bfloat16*>(vcache), v_tok, block_tables, max_blocks, bt_row, rows, ctx_len, block_size, n_q, n_kv,
        dk, dv, scale, window, chunk, softcap, sink, static_cast<__nv_bfloat16*>(out), o_head, o_row, ext);
  return static_cast<int>(cudaGetLastError());
}
