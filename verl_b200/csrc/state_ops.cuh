// Shared by the mixers that carry a state per sequence (delta rule, gated linear attention): vector loads, asynchronous copies,
// splits into bf16 terms, and the norm and gate of the heads' outputs.
#pragma once
#include "common.cuh"
#include "host_utils.h"

namespace vb {

template <typename T>
__device__ __forceinline__ float dl_f(T v) { return static_cast<float>(v); }
template <typename T>
__device__ __forceinline__ T dl_t(float v) { return static_cast<T>(v); }

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// For results that are rounded to bf16: the fast exponential and quotient err far below one bf16 ulp.
template <typename T>
__device__ __forceinline__ float silu_t(float x) {
  return sizeof(T) == 2 ? __fdividef(x, 1.f + __expf(-x)) : silu_f(x);
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// N consecutive elements, N * sizeof(T) aligned (N a power of two, at most 16 bytes at once).
template <typename T, int N>
__device__ __forceinline__ void load_n(const T* p, float (&f)[N]) {
  constexpr int W = sizeof(T) * N > 16 ? 16 / sizeof(T) : N;
  struct alignas(sizeof(T) * W) Vec { T v[W]; };
#pragma unroll
  for (int i = 0; i < N / W; ++i) {
    const Vec x = reinterpret_cast<const Vec*>(p)[i];
#pragma unroll
    for (int j = 0; j < W; ++j) f[i * W + j] = dl_f<T>(x.v[j]);
  }
}
template <typename T, int N>
__device__ __forceinline__ void store_n(T* p, const float (&f)[N]) {
  constexpr int W = sizeof(T) * N > 16 ? 16 / sizeof(T) : N;
  struct alignas(sizeof(T) * W) Vec { T v[W]; };
#pragma unroll
  for (int i = 0; i < N / W; ++i) {
    Vec x;
#pragma unroll
    for (int j = 0; j < W; ++j) x.v[j] = dl_t<T>(f[i * W + j]);
    reinterpret_cast<Vec*>(p)[i] = x;
  }
}

__device__ __forceinline__ void cp_async4(float* dst, const float* src, bool on) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 4 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}

__device__ __forceinline__ float sum8(float v) {  // over groups of eight lanes
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  return v;
}

// x = hi + lo, both bf16, for two neighbours packed into 32 bits
__device__ __forceinline__ void split2(float x0, float x1, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x0, x1);
  lo = pack_bf16x2(x0 - __uint_as_float(hi << 16), x1 - __uint_as_float(hi & 0xffff0000u));
}
struct GatedNormParams {
  void* out;         // [tokens, out_stride], first element of head 0
  long long out_stride;
  const void* gate;  // [tokens, stride], the same
  long long stride;
  const void* norm_w;  // [V]
  int H, V;
  float eps;
  bool vec;  // sizes, strides and addresses let four elements be read at once
};
// out = rmsnorm(out) * w * silu(gate) per (token, head), in place. A warp takes GN_T tokens of one head.
constexpr int GN_T = 4;
template <typename T>
__global__ void __launch_bounds__(128) gated_norm_kernel(const GatedNormParams p, int tokens) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (h >= p.H) return;
  const int t0 = blockIdx.x * GN_T, cnt = min(GN_T, tokens - t0);
  T* o = static_cast<T*>(p.out) + (long long)t0 * p.out_stride + (long long)h * p.V;
  const T* gate = static_cast<const T*>(p.gate) + (long long)t0 * p.stride + (long long)h * p.V;
  const T* w = static_cast<const T*>(p.norm_w);
  const float inv_v = 1.f / (float)p.V;
  const int c = lane * 4;
  if (p.V <= 128 && p.vec) {
    const bool on = c < p.V;
    float x[GN_T][4] = {}, g[GN_T][4], wv[4];
    if (on) load_n<T, 4>(w + c, wv);
#pragma unroll
    for (int k = 0; k < GN_T; ++k)
      if (on && k < cnt) {
        load_n<T, 4>(o + k * p.out_stride + c, x[k]);
        load_n<T, 4>(gate + k * p.stride + c, g[k]);
      }
#pragma unroll
    for (int k = 0; k < GN_T; ++k) {
      const float ss = x[k][0] * x[k][0] + x[k][1] * x[k][1] + x[k][2] * x[k][2] + x[k][3] * x[k][3];
      const float inv = rsqrtf(warp_reduce_sum(ss) * inv_v + p.eps);
      if (on && k < cnt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) x[k][e] = x[k][e] * inv * wv[e] * silu_t<T>(g[k][e]);
        store_n<T, 4>(o + k * p.out_stride + c, x[k]);
      }
    }
    return;
  }
  for (int k = 0; k < cnt; ++k, o += p.out_stride, gate += p.stride) {
    float ss = 0.f;
    for (int i = lane; i < p.V; i += 32) {
      const float x = dl_f<T>(o[i]);
      ss += x * x;
    }
    const float inv = rsqrtf(warp_reduce_sum(ss) * inv_v + p.eps);
    for (int i = lane; i < p.V; i += 32) o[i] = dl_t<T>(dl_f<T>(o[i]) * inv * dl_f<T>(w[i]) * silu_t<T>(dl_f<T>(gate[i])));
  }
}


template <typename T>
static int launch_gated_norm(T* out, long long out_stride, const T* gate, long long stride, const void* norm_w, int H, int V,
                             float eps, int tokens, cudaStream_t stream) {
  GatedNormParams p{out, out_stride, gate, stride, norm_w, H, V, eps, false};
  p.vec = V <= 128 && ((V | stride | out_stride) & 3) == 0 &&
          ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(gate)) & (4 * sizeof(T) - 1)) == 0;
  cudaError_t e = vb_launch_pdl(gated_norm_kernel<T>, dim3((tokens + GN_T - 1) / GN_T, (H + 3) / 4), dim3(128), 0, stream, 1, p,
                                tokens);
  vb_count_launch();
  return (int)e;
}

}  // namespace vb
