// Gated linear recurrent unit (ops/lru.py) over ragged batches with per-sequence state.
//
//   u = causal convolution of the recurrent branch (+ bias)              lru_conv
//   r, i = sigmoid(block-wise projections of u + bias)                   lru_gates (CUDA cores)
//   a = exp(-power r softplus(lam)),  v = sqrt(1 - a^2) i u
//   S = a S + v  token by token,  out = S gelu(gelu branch)              lru_scan (CUDA cores)
//
// Gates, decays and state are fp32. State [slots, W]; the convolution's inputs lie in a ring [slots, taps, W], position p in row
// p % taps. A sequence that starts at position 0 ignores what its slot held.
#include "host_utils.h"
#include "rowwise.cuh"

namespace vb {

struct LruParams {
  const int *cu_q, *seq_lens, *slots;
  int T, B, W, n, taps;  // n: channels of a block
  float power;
  long long stride;      // of proj rows: gelu branch (W) | recurrent branch (W)
  const float *gates_b, *lam;
  float* state;
};

// Sequence of token t.
__device__ __forceinline__ int seq_of(const int* __restrict__ cu_q, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// Decay a and input v of the recurrence from the gates' logits; c = -power * softplus(lam).
__device__ __forceinline__ void lru_terms(float zr, float zi, float u, float c, float& a, float& v) {
  const float la = c * sigmoid_f(zr);
  a = expf(la);
  v = sqrtf(-expm1f(2.f * la)) * sigmoid_f(zi) * u;
}

// u[t, c] = bias[c] + sum over j of x[t - taps + 1 + j, c] w[c, j]. Thread: V channels, LC_TOKENS tokens in a row. The row of a single
// token goes to its sequence's ring here; longer portions write theirs behind the scan (other tokens still read the ring).
constexpr int LC_TOKENS = 8;
template <typename T, int V>
__global__ void lru_conv_kernel(const T* __restrict__ proj, const T* __restrict__ w, const T* __restrict__ bias,
                                T* __restrict__ ring, T* __restrict__ u, const LruParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= p.W) return;
  const T* x = proj + p.W;
  const int t0 = blockIdx.x * LC_TOKENS, t1 = min(t0 + LC_TOKENS, p.T);
  int b = seq_of(p.cu_q, p.B, t0);
  for (int t = t0; t < t1; ++t) {
    while (p.cu_q[b + 1] <= t) ++b;
    const int first = p.cu_q[b], start = p.seq_lens[b] - (p.cu_q[b + 1] - first), slot = p.slots[b];
    float acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = to_f<T>(bias[c + e]);
    for (int j = 0; j < p.taps; ++j) {
      const int back = p.taps - 1 - j, at = t - back;  // row of the input, or (before the portion) position start + at - first
      float f[V];
      if (at >= first) {
        if constexpr (V == 8) ld8(x + at * p.stride + c, f); else f[0] = to_f<T>(x[at * p.stride + c]);
      } else {
        const int pos = start + at - first;
        if (pos < 0 || slot < 0) continue;
        const T* src = ring + ((long long)slot * p.taps + pos % p.taps) * p.W + c;
        if constexpr (V == 8) ld8(src, f); else f[0] = to_f<T>(src[0]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = fmaf(f[e], to_f<T>(w[(long long)(c + e) * p.taps + j]), acc[e]);
    }
    if constexpr (V == 8) st8(u + (long long)t * p.W + c, acc); else u[(long long)t * p.W + c] = from_f<T>(acc[0]);
    if (p.cu_q[b + 1] - first == 1 && slot >= 0) {
      T* dst = ring + ((long long)slot * p.taps + start % p.taps) * p.W + c;
#pragma unroll
      for (int e = 0; e < V; ++e) dst[e] = x[t * p.stride + c + e];
    }
  }
}

// The ring rows of a portion's last taps positions, for one channel (portions of two tokens up).
template <typename T>
__device__ __forceinline__ void write_ring(const T* __restrict__ x, T* __restrict__ ring, const LruParams& p, int first, int nq,
                                           int len, int slot, int c) {
  for (int pos = max(len - nq, len - p.taps); pos < len; ++pos)
    ring[((long long)slot * p.taps + pos % p.taps) * p.W + c] = x[(first + pos - (len - nq)) * p.stride + c];
}

// Decays and inputs [2, T, W] on the CUDA cores. One block per token and 128 channels.
template <typename T>
__global__ void lru_gates_kernel(const T* __restrict__ u, const T* __restrict__ gates, float* __restrict__ ab, const LruParams p) {
  extern __shared__ float row[];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) row[i] = to_f<T>(u[t * p.W + i]);
  __syncthreads();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.W) return;
  const int blk = c / p.n;
  const T *gr = gates + (long long)c * p.n, *gi = gr + (long long)p.W * p.n;
  const float* ub = row + blk * p.n;
  float zr = p.gates_b[c], zi = p.gates_b[p.W + c];
  for (int k = 0; k < p.n; ++k) {
    zr = fmaf(ub[k], to_f<T>(gr[k]), zr);
    zi = fmaf(ub[k], to_f<T>(gi[k]), zi);
  }
  float a, v;
  lru_terms(zr, zi, row[c], -p.power * softplus_f(p.lam[c]), a, v);
  ab[t * p.W + c] = a;
  ab[((long long)p.T + t) * p.W + c] = v;
}

// One thread per sequence and channel.
template <typename T>
__global__ void lru_scan_kernel(const T* __restrict__ proj, const float* __restrict__ ab, T* __restrict__ ring,
                                T* __restrict__ out, const LruParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c >= p.W) return;
  const int first = p.cu_q[b], nq = p.cu_q[b + 1] - first, len = p.seq_lens[b], slot = p.slots[b];
  const long long half = (long long)p.T * p.W;
  float S = slot >= 0 && len > nq ? p.state[(long long)slot * p.W + c] : 0.f;
  for (int t = first; t < first + nq; ++t) {
    const long long at = (long long)t * p.W + c;
    S = fmaf(ab[at], S, ab[half + at]);
    out[at] = from_f<T>(slot >= 0 ? S * gelu_tanh<sizeof(T) == 2>(to_f<T>(proj[t * p.stride + c])) : 0.f);
  }
  if (slot < 0 || nq <= 0) return;
  p.state[(long long)slot * p.W + c] = S;
  if (nq > 1) write_ring<T>(proj + p.W, ring, p, first, nq, len, slot, c);
}

}  // namespace vb

using namespace vb;
typedef __nv_bfloat16 bf16;

extern "C" int vb_rglru_tc_supported(int W, int n) { return 0; }

template <typename T>
static int rglru_simt(const void* proj, const void* conv_w, const void* conv_b, const void* gates, void* ring, void* u, float* ab,
                      void* out, const LruParams& p, bool tc, cudaStream_t stream) {
  const bool vec = (p.W & 7) == 0 && (p.stride & 7) == 0;
  const int v = vec ? 8 : 1, threads = p.W / v >= 256 ? 256 : 64;
  const dim3 g((p.T + LC_TOKENS - 1) / LC_TOKENS, (p.W / v + threads - 1) / threads);
  cudaError_t e;
  if (vec) e = vb_launch_pdl(lru_conv_kernel<T, 8>, g, dim3(threads), 0, stream, 1, (const T*)proj, (const T*)conv_w, (const T*)conv_b, (T*)ring, (T*)u, p);
  else e = vb_launch_pdl(lru_conv_kernel<T, 1>, g, dim3(threads), 0, stream, 1, (const T*)proj, (const T*)conv_w, (const T*)conv_b, (T*)ring, (T*)u, p);
  vb_count_launch();
  if (e != cudaSuccess || tc) return (int)e;
  e = vb_launch_pdl(lru_gates_kernel<T>, dim3(p.T, (p.W + 127) / 128), dim3(128), (size_t)p.W * 4, stream, 1, (const T*)u, (const T*)gates, ab, p);
  vb_count_launch();
  if (e != cudaSuccess) return (int)e;
  VB_DONE(vb_launch_pdl(lru_scan_kernel<T>, dim3((p.W + 63) / 64, p.B), dim3(64), 0, stream, 1, (const T*)proj, (const float*)ab, (T*)ring, (T*)out, p));
}

// proj [T, stride] (gelu branch | recurrent branch), conv_w [W, taps], gates [2, W / n, n, n], gates_b [2, W], lam [W] fp32, ring
// [slots, taps, W], state fp32 [slots, W], u [T, W] scratch, ab fp32 [2, T, W] scratch (without tc), out [T, W]. The leading
// `singles` sequences have one token each.
extern "C" int vb_rglru(const void* proj, long long stride, const void* conv_w, const void* conv_b, const void* gates,
                        const float* gates_b, const float* lam, void* ring, float* state, const int* cu_q, const int* seq_lens,
                        const int* slots, void* u, float* ab, void* out, int T, int B, int singles, int W, int n, int taps,
                        float power, int f32, int tc, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (W <= 0 || n <= 0 || W % n || taps <= 0 || B > 65535 || (W + 127) / 128 > 65535 || (size_t)W * 4 > 48 * 1024 || singles > B ||
      (!tc && ab == nullptr) || tc)
    return -3;
  LruParams p{cu_q, seq_lens, slots, T, B, W, n, taps, power, stride, gates_b, lam, state};
  return f32 ? rglru_simt<float>(proj, conv_w, conv_b, gates, ring, u, ab, out, p, false, stream)
             : rglru_simt<bf16>(proj, conv_w, conv_b, gates, ring, u, ab, out, p, false, stream);
}
