// Token-wise kernels of layer-list decoders (models/hybrid.py): 32-bit residual stream with fused add + RMSNorm, scaled
// embedding, clamped GLU, whole-projection query / key norm fused with the paged KV write, a CUDA-core matrix product for
// 32-bit weights (and for shapes that TMA cannot describe), and a CUDA-core paged attention that takes any head size.
//
// Every kernel is a template over the activation type (bf16 when serving, fp32 for the exact mode); arithmetic is fp32.
#include "common.cuh"
#include "host_utils.h"

namespace vb {

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// Eight consecutive elements (16-byte aligned).
__device__ __forceinline__ void ld8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 x = __bfloat1622float2(h[i]);
    f[2 * i] = x.x;
    f[2 * i + 1] = x.y;
  }
}
__device__ __forceinline__ void ld8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void st8(__nv_bfloat16* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]),
                                            pack_bf16x2(f[6], f[7]));
}
__device__ __forceinline__ void st8(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}

// Sum over the block, the same value in every thread. `sh` holds 32 floats.
__device__ __forceinline__ float block_sum_all(float v, float* sh) {
  v = warp_reduce_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (lane == 0) sh[warp] = v;
  __syncthreads();
  return warp_reduce_sum(lane < nw ? sh[lane] : 0.f);
}

// ---------------------------------------------------------------------------------------------------------------
// res[t] = table[ids[t]] * scale, fp32.
template <typename T>
__global__ void embed_scaled_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                                    float* __restrict__ res, int H, float scale) {
  pdl_trigger();
  pdl_wait();
  const T* src = table + ids[blockIdx.x] * (long long)H;
  float* dst = res + (long long)blockIdx.x * H;
  if ((H & 7) == 0) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8];
      ld8(src + v * 8, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] *= scale;
      st8(dst + v * 8, f);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = to_f<T>(src[i]) * scale;
  }
}

// ---------------------------------------------------------------------------------------------------------------
// res += delta (when given); y = res / sqrt(mean(res^2) + eps) * w. The residual stays fp32 in global memory; the row is
// kept in shared memory between the two passes.
template <typename T>
__global__ void add_rmsnorm_kernel(const T* __restrict__ delta, long long delta_stride, float* __restrict__ res,
                                   const T* __restrict__ w, T* __restrict__ y, int H, float eps) {
  extern __shared__ float row[];
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  float* r = res + (long long)blockIdx.x * H;
  T* out = y + (long long)blockIdx.x * H;
  const T* d = delta ? delta + (long long)blockIdx.x * delta_stride : nullptr;
  float ss = 0.f;
  const bool vec = (H & 7) == 0 && (d == nullptr || (delta_stride & 7) == 0);
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8];
      ld8(r + v * 8, f);
      if (d) {
        float g[8];
        ld8(d + v * 8, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += g[i];
        st8(r + v * 8, f);
      }
      st8(row + v * 8, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss += f[i] * f[i];
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      float f = r[i];
      if (d) {
        f += to_f<T>(d[i]);
        r[i] = f;
      }
      row[i] = f;
      ss += f * f;
    }
  }
  ss = block_sum_all(ss, sh);
  const float inv = 1.f / sqrtf(ss / (float)H + eps);
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {  // the same elements this thread has stored
      float f[8], g[8];
      ld8(row + v * 8, f);
      ld8(w + v * 8, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = f[i] * inv * g[i];
      st8(out + v * 8, f);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) out[i] = from_f<T>(row[i] * inv * to_f<T>(w[i]));
  }
}

// ---------------------------------------------------------------------------------------------------------------
// gu rows hold [gate (F) | up (F)]: g = min(gate, limit), u = clamp(up, -limit, limit), y = g sigmoid(alpha g) (u + 1).
template <typename T>
__device__ __forceinline__ float clamped_glu_1(float g, float u, float limit, float alpha) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  if (sizeof(T) == 2) return __fdividef(g, 1.f + __expf(-alpha * g)) * (u + 1.f);  // error far below a bf16 ulp
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}
template <typename T>
__global__ void clamped_glu_kernel(const T* __restrict__ gu, long long stride, T* __restrict__ y, long long total, int F,
                                   float limit, float alpha) {
  pdl_trigger();
  pdl_wait();
  const long long step = (long long)gridDim.x * blockDim.x;
  if ((F & 7) == 0 && (stride & 7) == 0) {
    const int nv = F >> 3;
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total / 8; i += step) {
      const long long t = i / nv;
      const int c = (int)(i - t * nv) * 8;
      float g[8], u[8];
      ld8(gu + t * stride + c, g);
      ld8(gu + t * stride + F + c, u);
#pragma unroll
      for (int k = 0; k < 8; ++k) g[k] = clamped_glu_1<T>(g[k], u[k], limit, alpha);
      st8(y + t * F + c, g);
    }
  } else {
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += step) {
      const long long t = i / F;
      const int c = (int)(i - t * F);
      y[i] = from_f<T>(clamped_glu_1<T>(to_f<T>(gu[t * stride + c]), to_f<T>(gu[t * stride + F + c]), limit, alpha));
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------
// One block per token. qkv row = [q (Hq * D) | k (Hk * D) | v (Hk * Dv)]. With norm weights: q and k are divided by the
// root mean square of the WHOLE projection (all heads together) and multiplied by their weights. q is normalised in
// place; k and v go to the token's place in the paged caches ([NB, Hk, BS, D] / [NB, Hk, BS, Dv]; slot < 0: no write).
template <typename T, bool VEC>
__global__ void qk_norm_kv_write_kernel(T* __restrict__ qkv, long long stride, const T* __restrict__ qw,
                                        const T* __restrict__ kw, const long long* __restrict__ slots,
                                        T* __restrict__ kc, T* __restrict__ vc, int Hq, int Hk, int D, int Dv,
                                        int block_size, float eps) {
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  T* q = qkv + (long long)blockIdx.x * stride;
  T* k = q + Hq * D;
  T* v = k + Hk * D;
  const int nq = Hq * D, nk = Hk * D, nv = Hk * Dv;
  constexpr int W = VEC ? 8 : 1;
  float iq = 1.f, ik = 1.f;
  if (qw != nullptr) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * W; i < nq + nk; i += blockDim.x * W) {  // q and k are adjacent
      float s = 0.f;
      if (VEC) {
        float f[8];
        ld8(q + i, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) s += f[e] * f[e];
      } else {
        const float f = to_f<T>(q[i]);
        s = f * f;
      }
      if (i < nq) sq += s; else sk += s;
    }
    sq = block_sum_all(sq, sh);
    sk = block_sum_all(sk, sh);
    iq = 1.f / sqrtf(sq / (float)nq + eps);
    ik = 1.f / sqrtf(sk / (float)nk + eps);
    for (int i = threadIdx.x * W; i < nq; i += blockDim.x * W) {
      if (VEC) {
        float f[8], g[8];
        ld8(q + i, f);
        ld8(qw + i, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = f[e] * iq * g[e];
        st8(q + i, f);
      } else {
        q[i] = from_f<T>(to_f<T>(q[i]) * iq * to_f<T>(qw[i]));
      }
    }
  }
  const long long slot = slots[blockIdx.x];
  if (slot < 0) return;
  const long long blk = slot / block_size, off = slot % block_size;
  for (int i = threadIdx.x * W; i < nk; i += blockDim.x * W) {
    const int h = i / D, d = i - h * D;
    T* dst = kc + ((blk * Hk + h) * block_size + off) * (long long)D + d;
    if (VEC) {
      float f[8], g[8];
      ld8(k + i, f);
      if (kw != nullptr) {
        ld8(kw + i, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = f[e] * ik * g[e];
      }
      st8(dst, f);
    } else {
      *dst = kw != nullptr ? from_f<T>(to_f<T>(k[i]) * ik * to_f<T>(kw[i])) : k[i];
    }
  }
  for (int i = threadIdx.x * W; i < nv; i += blockDim.x * W) {
    const int h = i / Dv, d = i - h * Dv;
    T* dst = vc + ((blk * Hk + h) * block_size + off) * (long long)Dv + d;
    if (VEC) {
      float f[8];
      ld8(v + i, f);
      st8(dst, f);
    } else {
      *dst = v[i];
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------
// C[M, N] = A[M, K] . B[N, K]^T (+ bias), fp32 accumulation on the CUDA cores. 64 x 64 tile, 4 x 4 per thread.
template <typename TA, typename TC>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const TA* __restrict__ A, const TA* __restrict__ B,
                                                        TC* __restrict__ C, const TA* __restrict__ bias, int M, int N,
                                                        int K, long long lda, long long ldb, long long ldc) {
  __shared__ float As[16][68], Bs[16][68];
  pdl_trigger();
  pdl_wait();
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256, r = e >> 4, c = e & 15;
      const bool ck = k0 + c < K;
      As[c][r] = (ck && m0 + r < M) ? to_f<TA>(A[(long long)(m0 + r) * lda + k0 + c]) : 0.f;
      Bs[c][r] = (ck && n0 + r < N) ? to_f<TA>(B[(long long)(n0 + r) * ldb + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 16; ++c) {
      const float4 a = *reinterpret_cast<const float4*>(&As[c][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Bs[c][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N)
        C[(long long)m * ldc + n] = from_f<TC>(acc[i][j] + (bias ? to_f<TA>(bias[n]) : 0.f));
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Paged attention over ragged queries on the CUDA cores: one warp per (token, query head), lanes across 32 keys for the
// scores and across the value dims for the weighted sum. A query at position i sees key j <= i when window <= 0, or
// i - j < window, or j < keep_first; bias[h][min(i - j, bias_len - 1)] is added to the scaled score.
struct PagedSimtParams {
  const int* cu_q;
  const int* seq_lens;
  const int* block_table;
  long long q_stride, out_stride;
  int max_blocks, B, Hq, Hk, D, Dv, block_size, window, keep_first, bias_len;
  float scale;
  const float* bias;
};
constexpr int PS_WARPS = 4, PS_MAX_D = 512, PS_VREG = PS_MAX_D / 32;

template <typename T>
__global__ void __launch_bounds__(PS_WARPS * 32)
paged_attn_simt_kernel(const T* __restrict__ q, const T* __restrict__ kc, const T* __restrict__ vc, T* __restrict__ out,
                       const PagedSimtParams p) {
  __shared__ float q_s[PS_WARPS][PS_MAX_D];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * PS_WARPS + warp, t = blockIdx.x;
  if (h >= p.Hq) return;
  int lo = 0, hi = p.B - 1;  // sequence of token t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int b = lo;
  const int pos = p.seq_lens[b] - (p.cu_q[b + 1] - t);
  const int hk = h / (p.Hq / p.Hk);
  const T* qr = q + (long long)t * p.q_stride + (long long)h * p.D;
  for (int d = lane; d < p.D; d += 32) q_s[warp][d] = to_f<T>(qr[d]);
  __syncwarp();
  const int* bt = p.block_table + (long long)b * p.max_blocks;
  const float* bias = p.bias ? p.bias + (long long)h * p.bias_len : nullptr;
  float m = -INFINITY, l = 0.f, acc[PS_VREG];
#pragma unroll
  for (int i = 0; i < PS_VREG; ++i) acc[i] = 0.f;
  const int n = pos + 1;
  const int w_lo = p.window > 0 ? max(0, n - p.window) : 0;      // first key of the window
  const int keep = min(p.window > 0 ? p.keep_first : 0, w_lo);   // kept keys in front of it
  const int total = keep + n - w_lo;
  for (int c = 0; c < total; c += 32) {
    const int idx = c + lane;
    const bool valid = idx < total;
    const int key = idx < keep ? idx : w_lo + idx - keep;
    long long row = 0;
    float s = -INFINITY;
    if (valid) {
      row = ((long long)bt[key / p.block_size] * p.Hk + hk) * p.block_size + key % p.block_size;
      const T* kr = kc + row * p.D;
      float a = 0.f;
      for (int d = 0; d < p.D; ++d) a = fmaf(q_s[warp][d], to_f<T>(kr[d]), a);
      s = a * p.scale;
      if (bias) s += bias[min(pos - key, p.bias_len - 1)];
    }
    const float nm = fmaxf(m, warp_reduce_max(s));
    const float alpha = expf(m - nm);
    const float w = valid ? expf(s - nm) : 0.f;
    l = l * alpha + warp_reduce_sum(w);
    m = nm;
#pragma unroll
    for (int i = 0; i < PS_VREG; ++i) acc[i] *= alpha;
    const int cnt = min(32, total - c);
    for (int j = 0; j < cnt; ++j) {
      const float wj = __shfl_sync(0xffffffffu, w, j);
      const T* vr = vc + __shfl_sync(0xffffffffu, row, j) * p.Dv;
#pragma unroll
      for (int i = 0; i < PS_VREG; ++i)
        if (lane + 32 * i < p.Dv) acc[i] = fmaf(wj, to_f<T>(vr[lane + 32 * i]), acc[i]);
    }
  }
  T* o = out + (long long)t * p.out_stride + (long long)h * p.Dv;
#pragma unroll
  for (int i = 0; i < PS_VREG; ++i)
    if (lane + 32 * i < p.Dv) o[lane + 32 * i] = from_f<T>(acc[i] / l);
}

}  // namespace vb

using namespace vb;
typedef __nv_bfloat16 bf16;

#define VB_DONE(e)                                   \
  do {                                               \
    cudaError_t _r = (e);                            \
    vb_count_launch();                               \
    return _r != cudaSuccess ? (int)_r : (int)cudaGetLastError(); \
  } while (0)

static inline int row_threads(int n) { return n >= 2048 ? 256 : (n >= 1024 ? 128 : 64); }

extern "C" int vb_embed_scaled(const long long* ids, const void* table, float* res, int T, int H, float scale, int f32,
                               cudaStream_t stream) {
  if (T <= 0) return 0;
  const dim3 g(T), b(row_threads(H));
  if (f32) VB_DONE(vb_launch_pdl(embed_scaled_kernel<float>, g, b, 0, stream, 1, ids, (const float*)table, res, H, scale));
  VB_DONE(vb_launch_pdl(embed_scaled_kernel<bf16>, g, b, 0, stream, 1, ids, (const bf16*)table, res, H, scale));
}

extern "C" int vb_add_rmsnorm(const void* delta, long long delta_stride, float* res, const void* w, void* y, int T, int H,
                              float eps, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  const size_t smem = (size_t)H * 4;
  if (smem > 160 * 1024) return -3;
  const dim3 g(T), b(row_threads(H));
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(add_rmsnorm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    VB_CUDA_CHECK(cudaFuncSetAttribute(add_rmsnorm_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    attr = true;
  }
  if (f32)
    VB_DONE(vb_launch_pdl(add_rmsnorm_kernel<float>, g, b, smem, stream, 1, (const float*)delta, delta_stride, res,
                          (const float*)w, (float*)y, H, eps));
  VB_DONE(vb_launch_pdl(add_rmsnorm_kernel<bf16>, g, b, smem, stream, 1, (const bf16*)delta, delta_stride, res,
                        (const bf16*)w, (bf16*)y, H, eps));
}

extern "C" int vb_clamped_glu(const void* gu, long long stride, void* y, int T, int F, float limit, float alpha, int f32,
                              cudaStream_t stream) {
  if (T <= 0 || F <= 0) return 0;
  const long long total = (long long)T * F;
  long long blocks = (total / 8 + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (blocks < 1) blocks = 1;
  const dim3 g((unsigned)blocks), b(256);
  if (f32)
    VB_DONE(vb_launch_pdl(clamped_glu_kernel<float>, g, b, 0, stream, 1, (const float*)gu, stride, (float*)y, total, F,
                          limit, alpha));
  VB_DONE(vb_launch_pdl(clamped_glu_kernel<bf16>, g, b, 0, stream, 1, (const bf16*)gu, stride, (bf16*)y, total, F, limit,
                        alpha));
}

// qw / kw null: no norm (q untouched, k and v only written to the cache).
extern "C" int vb_qk_norm_kv_write(void* qkv, long long stride, const void* qw, const void* kw, const long long* slots,
                                   void* kc, void* vc, int T, int Hq, int Hk, int D, int Dv, int block_size, float eps,
                                   int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((qw == nullptr) != (kw == nullptr)) return -3;
  const bool vec = (D & 7) == 0 && (Dv & 7) == 0 && (stride & 7) == 0;
  const dim3 g(T), b(row_threads(Hq * D));
#define VB_QKN(TT, V)                                                                                              \
  VB_DONE(vb_launch_pdl(qk_norm_kv_write_kernel<TT, V>, g, b, 0, stream, 1, (TT*)qkv, stride, (const TT*)qw,       \
                        (const TT*)kw, slots, (TT*)kc, (TT*)vc, Hq, Hk, D, Dv, block_size, eps))
  if (f32) {
    if (vec) VB_QKN(float, true);
    VB_QKN(float, false);
  }
  if (vec) VB_QKN(bf16, true);
  VB_QKN(bf16, false);
#undef VB_QKN
}

// a_f32 / out_f32: element types of (A, B, bias) and of C (fp32 inputs give fp32 outputs).
extern "C" int vb_gemm_simt(const void* A, const void* B, void* C, const void* bias, int M, int N, int K, long long lda,
                            long long ldb, long long ldc, int a_f32, int out_f32, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  if (K <= 0 || (M + 63) / 64 > 65535 || (a_f32 && !out_f32)) return -3;
  const dim3 g((N + 63) / 64, (M + 63) / 64), b(256);
  if (a_f32)
    VB_DONE(vb_launch_pdl(gemm_simt_kernel<float, float>, g, b, 0, stream, 1, (const float*)A, (const float*)B, (float*)C,
                          (const float*)bias, M, N, K, lda, ldb, ldc));
  if (out_f32)
    VB_DONE(vb_launch_pdl(gemm_simt_kernel<bf16, float>, g, b, 0, stream, 1, (const bf16*)A, (const bf16*)B, (float*)C,
                          (const bf16*)bias, M, N, K, lda, ldb, ldc));
  VB_DONE(vb_launch_pdl(gemm_simt_kernel<bf16, bf16>, g, b, 0, stream, 1, (const bf16*)A, (const bf16*)B, (bf16*)C,
                        (const bf16*)bias, M, N, K, lda, ldb, ldc));
}

extern "C" int vb_paged_attention_simt(const void* q, long long q_stride, const void* kc, const void* vc,
                                       const int* block_table, int max_blocks, const int* cu_q, const int* seq_lens,
                                       int T, int B, int Hq, int Hk, int D, int Dv, int block_size, float scale,
                                       int window, int keep_first, const float* bias, int bias_len, void* out,
                                       long long out_stride, int f32, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (Hk <= 0 || Hq % Hk != 0 || D <= 0 || D > PS_MAX_D || Dv <= 0 || Dv > PS_MAX_D || (bias && bias_len <= 0)) return -3;
  PagedSimtParams p{cu_q, seq_lens, block_table, q_stride, out_stride, max_blocks, B,          Hq,    Hk,  D,
                    Dv,   block_size, window,    keep_first, bias_len, scale,      bias};
  const dim3 g(T, (Hq + PS_WARPS - 1) / PS_WARPS), b(PS_WARPS * 32);
  if (f32)
    VB_DONE(vb_launch_pdl(paged_attn_simt_kernel<float>, g, b, 0, stream, 1, (const float*)q, (const float*)kc,
                          (const float*)vc, (float*)out, p));
  VB_DONE(vb_launch_pdl(paged_attn_simt_kernel<bf16>, g, b, 0, stream, 1, (const bf16*)q, (const bf16*)kc,
                        (const bf16*)vc, (bf16*)out, p));
}
