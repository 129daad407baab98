// Mixtures of experts when serving (ops/moe.py): choice of the experts by fp32 router logits, the layout of the buffer sorted
// by expert (every expert's rows padded to a multiple of 128, as the grouped GEMM wants them), the copy of the tokens into it,
// and the sum over a token's experts, fused with the residual add and the norm behind it. Nothing is read back to the host.
#include "host_utils.h"
#include "rowwise.cuh"

namespace vb {

constexpr int MR_MAX_E = 512, MR_MAX_TOP = 32, MR_BLK = 128;

struct MoeRouteParams {
  const float* logits;
  const float* correction;  // [E] or null: joins the scores for the choice
  long long stride;
  int T, E, top, softmax, renormalize, per_block, nblk;
  int *idx, *dest, *blk_expert;  // [T, top], [T, top], [nblk]
  float* weight;                 // [T, top]
  int* counters;                 // [E] pairs per expert, then a ticket; zero before and after
};

// Exclusive prefix sum of the experts' padded sizes (off_s[0 .. E]) by the first warp; counts in cnt_s.
__device__ __forceinline__ void padded_offsets(const int* cnt_s, int* off_s, int E) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    int run = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane;
      int v = e < E ? (cnt_s[e] + MR_BLK - 1) / MR_BLK * MR_BLK : 0;
      const int own = v;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += up;
      }
      if (e < E) off_s[e] = run + v - own;
      run += __shfl_sync(0xffffffffu, v, 31);
    }
    if (lane == 0) off_s[E] = run;
  }
}

// Expert of every block of 128 rows; -1 behind the last.
__device__ __forceinline__ void fill_blocks(const int* off_s, int E, int* blk_expert, int nblk) {
  for (int i = threadIdx.x; i < nblk; i += blockDim.x) {
    const int row = i * MR_BLK;
    int lo = 0, hi = E - 1;  // last expert that starts at or before the row; empty ones before it start there as well
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (off_s[mid] <= row) lo = mid; else hi = mid - 1;
    }
    blk_expert[i] = row < off_s[E] ? lo : -1;
  }
}

// One warp per token. NV = scores per lane.
template <int NV>
__global__ void __launch_bounds__(1024) moe_route_kernel(const MoeRouteParams p) {
  __shared__ int hist[MR_MAX_E], base[MR_MAX_E + 1];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  for (int e = threadIdx.x; e < p.E; e += blockDim.x) hist[e] = 0;
  __syncthreads();
  const int t0 = blockIdx.x * p.per_block, t1 = min(t0 + p.per_block, p.T);
  for (int t = t0 + warp; t < t1; t += warps) {
    const float* z = p.logits + t * p.stride;
    float s[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) s[i] = i * 32 + lane < p.E ? z[i * 32 + lane] : -INFINITY;
    if (p.softmax) {
      float m = -INFINITY, l = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) m = fmaxf(m, s[i]);
      m = warp_reduce_max(m);
#pragma unroll
      for (int i = 0; i < NV; ++i) l += s[i] = expf(s[i] - m);
      l = warp_reduce_sum(l);
#pragma unroll
      for (int i = 0; i < NV; ++i) s[i] /= l;
    } else {
#pragma unroll
      for (int i = 0; i < NV; ++i) s[i] = sigmoid_f(s[i]);
    }
    // scores are never negative: -1 for what is no number (chosen last). c: what the choice goes by, -inf for what is taken or
    // not there
    float c[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = i * 32 + lane;
      s[i] = s[i] >= 0.f ? s[i] : -1.f;
      c[i] = e >= p.E ? -INFINITY : s[i] + (p.correction && s[i] >= 0.f ? p.correction[e] : 0.f);
      if (e < p.E) c[i] = fmaxf(c[i], -3.0e38f);  // a correction that is no number, or minus infinity
    }
    int my_e = 0;
    float my_w = 0.f, total = 0.f;
    for (int k = 0; k < p.top; ++k) {
      float v = -INFINITY;
      int e = p.E;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (c[i] > v) {
          v = c[i];
          e = i * 32 + lane;
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oe = __shfl_xor_sync(0xffffffffu, e, o);
        if (ov > v || (ov == v && oe < e)) {
          v = ov;
          e = oe;
        }
      }
      float own = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (i * 32 + lane == e) {
          c[i] = -INFINITY;
          own = s[i];
        }
      v = __shfl_sync(0xffffffffu, own, e & 31);  // the score itself is the weight
      total += v;
      if (lane == k) {
        my_e = e;
        my_w = v;
      }
    }
    if (lane < p.top) {
      const long long at = (long long)t * p.top + lane;
      p.idx[at] = my_e;
      p.weight[at] = p.renormalize ? my_w / (total + 1e-20f) : my_w;
      p.dest[at] = atomicAdd(&hist[my_e], 1);
    }
  }
  __syncthreads();
  if (gridDim.x == 1) {  // the whole step: the layout as well
    padded_offsets(hist, base, p.E);
    __syncthreads();
    fill_blocks(base, p.E, p.blk_expert, p.nblk);
  } else {
    for (int e = threadIdx.x; e < p.E; e += blockDim.x) base[e] = hist[e] ? atomicAdd(&p.counters[e], hist[e]) : 0;
    __syncthreads();
  }
  for (int i = threadIdx.x; i < (t1 - t0) * p.top; i += blockDim.x) {
    const long long at = (long long)t0 * p.top + i;
    p.dest[at] += base[p.idx[at]];
  }
}

// Behind a route kernel of several blocks: places within the expert -> rows of the buffer.
__global__ void moe_layout_kernel(const MoeRouteParams p) {
  __shared__ int cnt[MR_MAX_E], off[MR_MAX_E + 1], last;
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e < p.E; e += blockDim.x) cnt[e] = __ldcg(&p.counters[e]);
  __syncthreads();
  padded_offsets(cnt, off, p.E);
  // the block that has read the counters last clears them
  if (threadIdx.x == 0) {
    __threadfence();
    last = atomicAdd(&p.counters[p.E], 1) == (int)gridDim.x - 1;
  }
  __syncthreads();
  if (last)
    for (int e = threadIdx.x; e <= p.E; e += blockDim.x) p.counters[e] = 0;
  if (blockIdx.x == 0) fill_blocks(off, p.E, p.blk_expert, p.nblk);
  const long long n = (long long)p.T * p.top, step = (long long)gridDim.x * blockDim.x;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += step) p.dest[i] += off[p.idx[i]];
}

// xs[dest[t, k]] = x[t], scale[dest[t, k]] = weight[t, k]. One block per token.
template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ x, long long stride, const int* __restrict__ dest,
                                  const float* __restrict__ weight, int top, int H, T* __restrict__ xs,
                                  float* __restrict__ scale) {
  __shared__ int to[MR_MAX_TOP];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  if (threadIdx.x < top) {
    const int d = dest[t * top + threadIdx.x];
    to[threadIdx.x] = d;
    scale[d] = weight[t * top + threadIdx.x];
  }
  __syncthreads();
  const T* src = x + t * stride;
  constexpr int W = 16 / sizeof(T);
  if (H % W == 0 && stride % W == 0) {
    for (int i = threadIdx.x; i < H / W; i += blockDim.x) {
      const uint4 v = reinterpret_cast<const uint4*>(src)[i];
      for (int k = 0; k < top; ++k) reinterpret_cast<uint4*>(xs + (long long)to[k] * H)[i] = v;
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x)
      for (int k = 0; k < top; ++k) xs[(long long)to[k] * H + i] = src[i];
  }
}

// d = sum over k of out[dest[t, k]] (* weight[t, k]) + shared[t] * sigmoid(logit[t]). Without post: res[t] += d,
// y = res / sqrt(mean + eps) * w, or without w the residual. With post: d *= sigmoid(gate[t]) element by element (when given),
// res += d / sqrt(mean(d^2) + eps) * post, y = res / sqrt(mean + eps) * w * scale. One block per token.
template <typename T>
__global__ void moe_combine_kernel(const T* __restrict__ out, const int* __restrict__ dest, const float* __restrict__ weight,
                                   int top, const T* __restrict__ shared, long long shared_stride,
                                   const float* __restrict__ logit, long long logit_stride, const T* __restrict__ gate,
                                   long long gate_stride, const T* __restrict__ post, float* __restrict__ res,
                                   const T* __restrict__ w, float scale, T* __restrict__ y, int H, float eps, bool vec) {
  extern __shared__ float row[];
  __shared__ float sh[32], wk[MR_MAX_TOP];
  __shared__ int from[MR_MAX_TOP];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  if (threadIdx.x < top) {
    from[threadIdx.x] = dest[t * top + threadIdx.x];
    wk[threadIdx.x] = weight ? weight[t * top + threadIdx.x] : 1.f;
  }
  __syncthreads();
  const float g = shared ? (logit ? sigmoid_f(logit[t * logit_stride]) : 1.f) : 0.f;
  const T* s = shared ? shared + t * shared_stride : nullptr;
  const T* gt = gate ? gate + t * gate_stride : nullptr;
  float* r = res + t * H;
  float ss = 0.f;
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float a[8] = {}, f[8];
      if (!post) ld8(r + v * 8, a);
      if (s) {
        ld8(s + v * 8, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) a[i] = fmaf(f[i], g, a[i]);
      }
      for (int k = 0; k < top; ++k) {
        ld8(out + (long long)from[k] * H + v * 8, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) a[i] = fmaf(f[i], wk[k], a[i]);
      }
      if (gt) {
        ld8(gt + v * 8, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) a[i] *= sigmoid_t<T>(f[i]);
      }
      if (!post) st8(r + v * 8, a);
      st8(row + v * 8, a);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss += a[i] * a[i];
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      float a = post ? 0.f : r[i];
      if (s) a = fmaf(to_f<T>(s[i]), g, a);
      for (int k = 0; k < top; ++k) a = fmaf(to_f<T>(out[(long long)from[k] * H + i]), wk[k], a);
      if (gt) a *= sigmoid_t<T>(to_f<T>(gt[i]));
      row[i] = a;
      if (!post) r[i] = a;
      ss += a * a;
    }
  }
  if (post) norm_row_add(row, ss, r, post, w, scale, y + t * H, H, eps, vec, sh);
  else norm_row_out(row, ss, w, y + t * H, H, eps, vec, sh);
}

}  // namespace vb

using namespace vb;
typedef __nv_bfloat16 bf16;

// logits fp32 [T, stride], the first E of a row; idx, weight, dest [T, top]; blk_expert [nblk], nblk * 128 rows being enough for
// every expert's share rounded up to 128; counters [E + 1], zero before and after.
extern "C" int vb_moe_route(const float* logits, long long stride, int T, int E, int top, int softmax, int renormalize,
                            const float* correction, int* idx, float* weight, int* dest, int* blk_expert, int nblk, int* counters, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (E <= 0 || E > MR_MAX_E || top <= 0 || top > MR_MAX_TOP || top > E ||
      (long long)nblk * MR_BLK + MR_BLK <= (long long)T * top + (long long)min(E, T * top) * (MR_BLK - 1))
    return -3;
  const bool small = T <= 32;
  const int per = small ? T : (T <= 4096 ? 8 : 64);
  MoeRouteParams p{logits, correction, stride, T, E, top, softmax, renormalize, per, nblk, idx, dest, blk_expert, weight, counters};
  const dim3 g((T + per - 1) / per), b(small ? (T + 3) / 4 * 128 : 256);
#define VB_MR(NV) e = vb_launch_pdl(moe_route_kernel<NV>, g, b, 0, stream, 1, p)
  cudaError_t e;
  if (E <= 32) VB_MR(1);
  else if (E <= 64) VB_MR(2);
  else if (E <= 128) VB_MR(4);
  else if (E <= 256) VB_MR(8);
  else VB_MR(16);
#undef VB_MR
  vb_count_launch();
  if (e != cudaSuccess) return (int)e;
  if (small) return (int)cudaGetLastError();
  const long long n = (long long)T * top;
  VB_DONE(vb_launch_pdl(moe_layout_kernel, dim3((unsigned)min((n + 255) / 256, 296ll)), dim3(256), 0, stream, 1, p));
}

extern "C" int vb_moe_gather(const void* x, long long stride, const int* dest, const float* weight, int T, int top, int H, void* xs,
                             float* scale, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (top <= 0 || top > MR_MAX_TOP) return -3;
  const dim3 g(T), b(H >= 2048 ? 256 : 128);
  if (f32)
    VB_DONE(vb_launch_pdl(moe_gather_kernel<float>, g, b, 0, stream, 1, (const float*)x, stride, dest, weight, top, H, (float*)xs,
                          scale));
  VB_DONE(vb_launch_pdl(moe_gather_kernel<bf16>, g, b, 0, stream, 1, (const bf16*)x, stride, dest, weight, top, H, (bf16*)xs,
                        scale));
}

// weight null: the rows of out are added as they are. shared null: none; logit null: its factor is one. post, gate, scale: see
// moe_combine_kernel.
extern "C" int vb_moe_sum(const void* out, const int* dest, const float* weight, int top, const void* shared,
                          long long shared_stride, const float* logit, long long logit_stride, const void* gate,
                          long long gate_stride, const void* post, float* res, const void* w, float scale, void* y, int T, int H,
                          float eps, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  const size_t smem = (size_t)H * 4;
  if (smem > 160 * 1024 || top <= 0 || top > MR_MAX_TOP || (gate && !post)) return -3;
  const bool vec = ((H | shared_stride | gate_stride) & 7) == 0 &&
                   ((reinterpret_cast<uintptr_t>(shared) | reinterpret_cast<uintptr_t>(gate)) & 15) == 0;
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(moe_combine_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    VB_CUDA_CHECK(cudaFuncSetAttribute(moe_combine_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    attr = true;
  }
  const dim3 g(T), b(row_threads(H));
  if (f32)
    VB_DONE(vb_launch_pdl(moe_combine_kernel<float>, g, b, smem, stream, 1, (const float*)out, dest, weight, top,
                          (const float*)shared, shared_stride, logit, logit_stride, (const float*)gate, gate_stride,
                          (const float*)post, res, (const float*)w, scale, (float*)y, H, eps, vec));
  VB_DONE(vb_launch_pdl(moe_combine_kernel<bf16>, g, b, smem, stream, 1, (const bf16*)out, dest, weight, top, (const bf16*)shared,
                        shared_stride, logit, logit_stride, (const bf16*)gate, gate_stride, (const bf16*)post, res,
                        (const bf16*)w, scale, (bf16*)y, H, eps, vec));
}
