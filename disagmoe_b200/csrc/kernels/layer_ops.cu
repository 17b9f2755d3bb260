// Row kernels of decoders whose residual stream is kept in fp32, for bf16 and fp32 activations: scaled embedding,
// post-norm + residual add + pre-norm in one pass, per-head query / key norm + partial rotary embedding + paged KV
// append, rotary table from arbitrary frequencies, silu(gate) * up, and a CUDA-core GEMM for fp32 operands (and for bf16
// shapes the tcgen05 kernel's TMA cannot address).
#include "dmoe_kernels.h"
#include "sm100.cuh"

namespace dmoe {

typedef __nv_bfloat16 bf16;

template <typename T, int VEC>
struct Pack;   // VEC elements of T <-> floats, one aligned access where VEC > 1
template <typename T>
struct Pack<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float* f) { f[0] = static_cast<float>(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float* f) { p[0] = static_cast<T>(f[0]); }
};
template <>
struct Pack<float, 8> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
  }
};
template <>
struct Pack<bf16, 8> {
  static __device__ __forceinline__ void load(const bf16* p, float* f) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 t = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
      f[2 * i] = t.x;
      f[2 * i + 1] = t.y;
    }
  }
  static __device__ __forceinline__ void store(bf16* p, const float* f) {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 t = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
      w[i] = *reinterpret_cast<const uint32_t*>(&t);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
};

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

// out[t] = table[ids[t]] * scale, fp32
template <typename T>
__global__ void embed_f32_kernel(const int* __restrict__ ids, const T* __restrict__ table, float scale,
                                 float* __restrict__ out, int W, int vocab) {
  const long long t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) id = 0;
  const T* src = table + static_cast<long long>(id) * W;
  for (int i = threadIdx.x; i < W; i += blockDim.x) out[t * W + i] = static_cast<float>(src[i]) * scale;
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

// table[pos][i] = (cos, sin)(pos * freq[i]) * mscale, angles and functions in double precision
__global__ void rope_freq_table_kernel(float2* __restrict__ table, int max_pos, int half, const double* __restrict__ freq,
                                       float mscale) {
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= static_cast<long long>(max_pos) * half) return;
  double s, c;
  sincos(static_cast<double>(i / half) * freq[i % half], &s, &c);
  table[i] = make_float2(static_cast<float>(c * mscale), static_cast<float>(s * mscale));
}

// rows [q heads | k heads | v heads] (the last two only where n_kv > 0): RMS norm over each q / k head with its weight,
// rotation of the pairs (i, i + rot / 2), i < rot / 2, q written back in place, k and v appended to the paged caches
// ([blocks, block_size, n_kv, dk] and [.., dv]) at slots[t] (< 0: skip). One warp per head.
template <typename T>
__global__ void __launch_bounds__(256)
qk_norm_rope_kernel(T* __restrict__ qkv, long long ld, const int* __restrict__ positions,
                    const long long* __restrict__ slots, T* __restrict__ kcache, T* __restrict__ vcache, int n_q, int n_kv,
                    int dk, int dv, int rot, const float2* __restrict__ table, int max_pos, const float* __restrict__ qw,
                    const float* __restrict__ kw, float eps) {
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
    float ss = 0.f;
    for (int d = lane; d < dk; d += 32) {
      const float x = static_cast<float>(p[d]);
      ss += x * x;
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(dk) + eps);
    for (int i = lane; i < half; i += 32) {
      const float u = static_cast<float>(p[i]) * inv * w[i], v = static_cast<float>(p[i + half]) * inv * w[i + half];
      const float2 cs = tab[i];
      dst[i] = static_cast<T>(u * cs.x - v * cs.y);
      dst[i + half] = static_cast<T>(v * cs.x + u * cs.y);
    }
    for (int d = rot + lane; d < dk; d += 32) dst[d] = static_cast<T>(static_cast<float>(p[d]) * inv * w[d]);
  }
  if (slot >= 0) {
    const T* src = row + static_cast<long long>(n_q + n_kv) * dk;
    T* dst = vcache + slot * n_kv * dv;
    for (int i = threadIdx.x; i < n_kv * dv; i += blockDim.x) dst[i] = src[i];
  }
}

// out[t, i] = silu(gu[t, i]) * gu[t, I + i]
template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gu, long long ld, T* __restrict__ out, long long ld_out, int I) {
  const long long t = blockIdx.y;
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= I) return;
  const float g = static_cast<float>(gu[t * ld + i]), u = static_cast<float>(gu[t * ld + I + i]);
  out[t * ld_out + i] = static_cast<T>(g / (1.f + expf(-g)) * u);
}

// Y[t, f] = sum_k X[t, k] W[f, k] with fp32 multiply-adds: 64 x 64 tiles, 4 x 4 outputs per thread.
constexpr int kSgTile = 64, kSgK = 16;

template <typename T, typename TY>
__global__ void __launch_bounds__(256)
simt_gemm_kernel(const T* __restrict__ X, long long ldx, const T* __restrict__ W, long long ldw, TY* __restrict__ Y,
                 long long ldy, int M, int F, int K) {
  __shared__ float sx[kSgK][kSgTile + 4], sw[kSgK][kSgTile + 4];
  const int t0 = blockIdx.y * kSgTile, f0 = blockIdx.x * kSgTile;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kSgK) {
    for (int i = threadIdx.x; i < kSgTile * kSgK; i += 256) {
      const int r = i / kSgK, k = i % kSgK;
      const bool in_k = k0 + k < K;
      sx[k][r] = in_k && t0 + r < M ? static_cast<float>(X[(t0 + r) * ldx + k0 + k]) : 0.f;
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
    if (t >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int f = f0 + tx * 4 + j;
      if (f < F) Y[t * ldy + f] = static_cast<TY>(acc[i][j]);
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

}  // namespace dmoe

using namespace dmoe;

extern "C" int dmoe_embed_f32(const int* ids, const void* table, int is_f32, float scale, float* out, int T, int W, int vocab,
                              void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (W < 1 || vocab < 1) return -10;
  if (T == 0) return 0;
  const int threads = W >= 256 ? 256 : 64;
  if (is_f32)
    embed_f32_kernel<float><<<T, threads, 0, stream>>>(ids, static_cast<const float*>(table), scale, out, W, vocab);
  else
    embed_f32_kernel<bf16><<<T, threads, 0, stream>>>(ids, static_cast<const bf16*>(table), scale, out, W, vocab);
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

extern "C" int dmoe_qk_norm_rope(int is_f32, void* qkv, long long ld, const int* positions, const long long* slots,
                                 void* kcache, void* vcache, int T, int n_q, int n_kv, int dk, int dv, int rot,
                                 const void* table, int max_pos, const float* qw, const float* kw, float eps, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (n_q < 1 || n_kv < 0 || dk < 1 || rot < 0 || rot % 2 != 0 || rot > dk || (rot > 0 && table == nullptr)) return -10;
  if (n_kv > 0 && (kcache == nullptr || vcache == nullptr || kw == nullptr)) return -10;
  if (T == 0) return 0;
  int threads = (n_q + n_kv) * 32;
  if (threads > 256) threads = 256;
  if (is_f32)
    qk_norm_rope_kernel<float><<<T, threads, 0, stream>>>(
        static_cast<float*>(qkv), ld, positions, slots, static_cast<float*>(kcache), static_cast<float*>(vcache), n_q, n_kv,
        dk, dv, rot, static_cast<const float2*>(table), max_pos, qw, kw, eps);
  else
    qk_norm_rope_kernel<bf16><<<T, threads, 0, stream>>>(
        static_cast<bf16*>(qkv), ld, positions, slots, static_cast<bf16*>(kcache), static_cast<bf16*>(vcache), n_q, n_kv, dk,
        dv, rot, static_cast<const float2*>(table), max_pos, qw, kw, eps);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_silu_mul(int is_f32, const void* gu, long long ld, void* out, long long ld_out, int T, int I,
                             void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (I < 1) return -10;
  for (int t0 = 0; t0 < T; t0 += 65535) {      // grid.y limit
    const int n = T - t0 < 65535 ? T - t0 : 65535;
    const dim3 grid((I + 255) / 256, n);
    if (is_f32)
      silu_mul_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const float*>(gu) + t0 * ld, ld,
                                                       static_cast<float*>(out) + t0 * ld_out, ld_out, I);
    else
      silu_mul_kernel<bf16><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(gu) + t0 * ld, ld,
                                                      static_cast<bf16*>(out) + t0 * ld_out, ld_out, I);
  }
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dmoe_simt_linear(int x_f32, int y_f32, const void* X, long long ldx, const void* W, long long ldw, void* Y,
                                long long ldy, int T, int F, int K, void* stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (F < 1 || K < 1 || (x_f32 && !y_f32)) return -10;
  if (T == 0) return 0;
  const long long ty = (T + kSgTile - 1) / kSgTile;
  if (ty > 65535) return -10;
  const dim3 grid((F + kSgTile - 1) / kSgTile, static_cast<unsigned>(ty));
  if (x_f32)
    simt_gemm_kernel<float, float><<<grid, 256, 0, stream>>>(static_cast<const float*>(X), ldx, static_cast<const float*>(W),
                                                             ldw, static_cast<float*>(Y), ldy, T, F, K);
  else if (y_f32)
    simt_gemm_kernel<bf16, float><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(X), ldx, static_cast<const bf16*>(W), ldw,
                                                            static_cast<float*>(Y), ldy, T, F, K);
  else
    simt_gemm_kernel<bf16, bf16><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(X), ldx, static_cast<const bf16*>(W), ldw,
                                                           static_cast<bf16*>(Y), ldy, T, F, K);
  return static_cast<int>(cudaGetLastError());
}
