// Shared by the token-wise kernels of layer-list decoders: templates over the activation type (bf16 when serving, fp32 for the
// exact mode) with fp32 arithmetic, eight elements at a time where alignment allows it.
#pragma once
#include "common.cuh"

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

// The row in shared memory, of which every thread has stored the elements it reads here: out = row / sqrt(mean + eps) * w, or
// without w the row. ss: this thread's sum of squares.
template <typename T>
__device__ __forceinline__ void norm_row_out(const float* row, float ss, const T* __restrict__ w, T* __restrict__ out, int H,
                                             float eps, bool vec, float* sh) {
  const float inv = w ? 1.f / sqrtf(block_sum_all(ss, sh) / (float)H + eps) : 1.f;
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8], g[8];
      ld8(row + v * 8, f);
      if (w) {
        ld8(w + v * 8, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = f[i] * inv * g[i];
      }
      st8(out + v * 8, f);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) out[i] = from_f<T>(w ? row[i] * inv * to_f<T>(w[i]) : row[i]);
  }
}

// The row in shared memory, of which every thread has stored the elements it reads here, with the sum of squares ss of this
// thread's: res += row / sqrt(mean(row^2) + eps) * w; out = res, or with fw: res / sqrt(mean(res^2) + eps) * fw * fscale.
template <typename T>
__device__ __forceinline__ void norm_row_add(float* row, float ss, float* __restrict__ res, const T* __restrict__ w,
                                             const T* __restrict__ fw, float fscale, T* __restrict__ out, int H, float eps,
                                             bool vec, float* sh) {
  const float inv = 1.f / sqrtf(block_sum_all(ss, sh) / (float)H + eps);
  ss = 0.f;
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8], g[8], x[8];
      ld8(res + v * 8, x);
      ld8(row + v * 8, f);
      ld8(w + v * 8, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        x[i] += f[i] * inv * g[i];
        ss += x[i] * x[i];
      }
      st8(res + v * 8, x);
      if (fw) st8(row + v * 8, x); else st8(out + v * 8, x);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float x = res[i] + row[i] * inv * to_f<T>(w[i]);
      res[i] = x;
      ss += x * x;
      if (fw) row[i] = x; else out[i] = from_f<T>(x);
    }
  }
  if (fw == nullptr) return;
  const float fi = fscale / sqrtf(block_sum_all(ss, sh) / (float)H + eps);
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8], g[8];
      ld8(row + v * 8, f);
      ld8(fw + v * 8, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = f[i] * fi * g[i];
      st8(out + v * 8, f);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) out[i] = from_f<T>(row[i] * fi * to_f<T>(fw[i]));
  }
}

// 1 / (1 + e^-z) for the activation type: errors far below a bf16 ulp are let through.
template <typename T>
__device__ __forceinline__ float sigmoid_t(float z) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z));
}

// gelu with tanh: 0.5 g (1 + tanh(z)) = g sigmoid(2 z), z = sqrt(2 / pi) (g + 0.044715 g^3). FAST: error far below a bf16 ulp.
template <bool FAST>
__device__ __forceinline__ float gelu_tanh(float g) {
  const float z = 0.7978845608028654f * (g + 0.044715f * g * g * g);
  if (FAST) return __fdividef(g, 1.f + __expf(-2.f * z));
  return 0.5f * g * (1.f + tanhf(z));
}
// gelu with erf: z Phi(z). FAST: erf by formula 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions (largest error
// 1.5e-7).
template <bool FAST>
__device__ __forceinline__ float gelu_erf(float z) {
  const float x = z * 0.70710678118654752f;
  if (!FAST) return 0.5f * z * (1.f + erff(x));
  const float a = fabsf(x), t = __fdividef(1.f, fmaf(0.3275911f, a, 1.f));
  const float y = t * fmaf(t, fmaf(t, fmaf(t, fmaf(t, 1.061405429f, -1.453152027f), 1.421413741f), -0.284496736f), 0.254829592f);
  const float tail = 0.5f * y * __expf(-a * a);  // 1 - Phi(|z|)
  return z * (z < 0.f ? tail : 1.f - tail);
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

}  // namespace vb

// Returns from a launcher with the launch's error, or the last one.
#define VB_DONE(e)                                   \
  do {                                               \
    cudaError_t _r = (e);                            \
    vb_count_launch();                               \
    return _r != cudaSuccess ? (int)_r : (int)cudaGetLastError(); \
  } while (0)

static inline int row_threads(int n) { return n >= 2048 ? 256 : (n >= 1024 ? 128 : 64); }
