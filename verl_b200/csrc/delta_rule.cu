// Gated delta rule over ragged batches with carried state (linear-attention mixer of layer-list decoders).
//
// Per head with state S [D, V], unit-norm k, scaled unit-norm q, decay g = exp(-exp(A_log) softplus(a + dt_bias)) and step
// beta = sigmoid(b):
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// and the head's output is rmsnorm(o) * w * silu(gate). q, k, v come from projections that pass a short causal
// convolution per channel and a silu.
//
// Input row of a token (one projection GEMM): [q (Hk D) | k (Hk D) | v (H V) | gate (H V) | b (H) | a (H)].
// State of a sequence (slot s): fp32 state[s][H][V][D] (a column of S is contiguous), and conv[s][taps][C] of the
// activation type, C = 2 Hk D + H V: a ring of the last `taps` convolution inputs, position p lives in row p % taps. A
// token overwrites the row of position p - taps, which no later token reads, so the kernel that handles one token may
// read and write the ring without ordering between its blocks. A sequence whose first token has position 0 starts from
// zero state whatever its slot holds; slot < 0 marks a padding row.
//
// Kernels: delta_prep (convolution, silu, unit norms, gates of every token) -> delta_scan (state carried through the
// tokens in registers, fp32) -> gated_norm; delta_step does all of it for sequences that bring one token each.
#include "common.cuh"
#include "host_utils.h"

namespace vb {

template <typename T>
__device__ __forceinline__ float dl_f(T v) { return static_cast<float>(v); }
template <typename T>
__device__ __forceinline__ T dl_t(float v) { return static_cast<T>(v); }

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
constexpr float UNIT_EPS = 1e-6f;

struct DeltaParams {
  const void* proj;        // [T, stride]
  long long stride;
  const void* conv_w;      // [C, taps]
  const float* a_log;      // [H]
  const float* dt_bias;    // [H]
  const void* norm_w;      // [V]
  void* ring;              // [slots, taps, C]
  float* state;            // [slots, H, V, D]
  const int* cu_q;         // [B + 1]
  const int* seq_lens;     // [B] tokens of the sequence up to and including this step's
  const int* slots;        // [B]
  float* qkv;              // [T, C] fp32 (scan path)
  float* gates;            // [T, 2 H] fp32: beta | log decay (scan path)
  void* out;               // [T, out_stride]
  long long out_stride;
  int B, H, Hk, D, V, taps;
  float eps;
};

// ---------------------------------------------------------------------------------------------------------------
// One warp per (sequence, tile of tokens, head row); lanes across the head's channels, a sliding window of inputs in
// registers. Head rows: Hk of q, Hk of k, H of v; one more row does the gates.
constexpr int DP_TT = 32;  // tokens per tile
template <typename T, int TAPS, int CPL>
__global__ void __launch_bounds__(128) delta_prep_kernel(const DeltaParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, r = blockIdx.y * 4 + (threadIdx.x >> 5), b = blockIdx.z;
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first;
  const int t0 = blockIdx.x * DP_TT, t1 = min(n, t0 + DP_TT);
  const int slot = p.slots[b], rows = 2 * p.Hk + p.H;
  if (t0 >= n || r > rows || slot < 0) return;
  const int start = p.seq_lens[b] - n;
  const int C = 2 * p.Hk * p.D + p.H * p.V;
  const T* proj = static_cast<const T*>(p.proj) + (long long)first * p.stride;
  if (r == rows) {
    for (int i = lane; i < (t1 - t0) * p.H; i += 32) {
      const int t = t0 + i / p.H, h = i % p.H;
      const T* row = proj + (long long)t * p.stride + C + p.H * p.V;
      float* g = p.gates + (long long)(first + t) * 2 * p.H;
      g[h] = sigmoid_f(dl_f<T>(row[h]));
      g[p.H + h] = -expf(p.a_log[h]) * softplus_f(dl_f<T>(row[p.H + h]) + p.dt_bias[h]);
    }
    return;
  }
  const bool qk = r < 2 * p.Hk;
  const int size = qk ? p.D : p.V, c0 = qk ? r * p.D : 2 * p.Hk * p.D + (r - 2 * p.Hk) * p.V;
  const T* ring = static_cast<const T*>(p.ring) + (long long)slot * p.taps * C + c0;
  const T* cw = static_cast<const T*>(p.conv_w) + (long long)c0 * p.taps;
  // w[j], hist[j]: tap and input of the token j places back; taps beyond p.taps stay zero
  float w[TAPS][CPL], hist[TAPS][CPL];
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      const int c = lane + 32 * i, t = t0 - j;
      const bool on = c < size && j < p.taps;
      w[j][i] = on ? dl_f<T>(cw[c * p.taps + p.taps - 1 - j]) : 0.f;
      float x = 0.f;
      if (on && j > 0) {
        if (t >= 0) x = dl_f<T>(proj[(long long)t * p.stride + c0 + c]);
        else if (start + t >= 0) x = dl_f<T>(ring[(long long)((start + t) % p.taps) * C + c]);
      }
      hist[j][i] = x;
    }
  const float qscale = r < p.Hk ? 1.f / sqrtf((float)p.D) : 1.f;
  for (int t = t0; t < t1; ++t) {
    float y[CPL], ss = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      const int c = lane + 32 * i;
      hist[0][i] = c < size ? dl_f<T>(proj[(long long)t * p.stride + c0 + c]) : 0.f;
      float a = 0.f;
#pragma unroll
      for (int j = TAPS - 1; j >= 0; --j) a = fmaf(w[j][i], hist[j][i], a);
#pragma unroll
      for (int j = TAPS - 1; j > 0; --j) hist[j][i] = hist[j - 1][i];
      y[i] = silu_f(a);
      ss += y[i] * y[i];  // channels past the head give silu(0) = 0
    }
    float mul = 1.f;
    if (qk) mul = qscale / sqrtf(warp_reduce_sum(ss) + UNIT_EPS);
    float* dst = p.qkv + (long long)(first + t) * C + c0;
#pragma unroll
    for (int i = 0; i < CPL; ++i)
      if (lane + 32 * i < size) dst[lane + 32 * i] = y[i] * mul;
  }
}

__device__ __forceinline__ void cp_async4(float* dst, const float* src, bool on) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 4 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float sum8(float v) {  // over groups of eight lanes
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  return v;
}

// ---------------------------------------------------------------------------------------------------------------
// One CTA per (sequence, head, 32 state columns). Eight lanes share a column; lane r holds rows 4 (r + 8 i) + e. Tokens
// come through a double-buffered shared-memory stage. Both products of a token use the old state (S^T k and S^T q in one
// pass): o = g S^T q + (k . q) u, so a token costs one reduction round.
constexpr int DS_VB = 32, DS_TB = 16, DS_THREADS = 256;
template <typename T, int NR>
__global__ void __launch_bounds__(DS_THREADS) delta_scan_kernel(const DeltaParams p) {
  constexpr int DP = NR * 8;
  extern __shared__ float sm[];
  float* k_s = sm;                            // [2][TB][DP]
  float* q_s = k_s + 2 * DS_TB * DP;          // [2][TB][DP]
  float* v_s = q_s + 2 * DS_TB * DP;          // [2][TB][VB]
  float* g_s = v_s + 2 * DS_TB * DS_VB;       // [2][TB][2] beta, log decay
  float* kq_s = g_s + 2 * DS_TB * 2;          // [TB]
  float* dec_s = kq_s + DS_TB;                // [TB]
  float* o_s = dec_s + DS_TB;                 // [TB][VB]
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, v0 = blockIdx.y * DS_VB, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane & 7, col = warp * 4 + (lane >> 3);
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;
  const int start = p.seq_lens[b] - n, hk = h / (p.H / p.Hk);
  const int C = 2 * p.Hk * p.D + p.H * p.V;
  const bool col_on = v0 + col < p.V;
  float* st = p.state + (((long long)slot * p.H + h) * p.V + v0 + col) * p.D;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = 4 * (r + 8 * (i >> 2)) + (i & 3);
    S[i] = (start > 0 && col_on && row < p.D) ? st[row] : 0.f;
  }
  const float* qkv = p.qkv + (long long)first * C;
  const float* gates = p.gates + (long long)first * 2 * p.H;
  auto stage = [&](int blk) {
    const int buf = blk & 1, t0 = blk * DS_TB;
    for (int i = tid; i < DS_TB * DP; i += DS_THREADS) {
      const int t = i / DP, d = i % DP;
      const bool on = t0 + t < n && d < p.D;
      const float* src = qkv + (long long)(on ? t0 + t : 0) * C + hk * p.D + (on ? d : 0);
      cp_async4(q_s + buf * DS_TB * DP + i, src, on);
      cp_async4(k_s + buf * DS_TB * DP + i, src + p.Hk * p.D, on);
    }
    for (int i = tid; i < DS_TB * DS_VB; i += DS_THREADS) {
      const int t = i / DS_VB, c = i % DS_VB;
      const bool on = t0 + t < n && v0 + c < p.V;
      cp_async4(v_s + buf * DS_TB * DS_VB + i,
                qkv + (on ? (long long)(t0 + t) * C + 2 * p.Hk * p.D + h * p.V + v0 + c : 0), on);
    }
    if (tid < DS_TB * 2) {
      const bool on = t0 + (tid >> 1) < n;
      cp_async4(g_s + buf * DS_TB * 2 + tid, gates + (on ? (long long)(t0 + (tid >> 1)) * 2 * p.H + (tid & 1) * p.H + h : 0), on);
    }
    cp_async_commit();
  };
  const int blocks = (n + DS_TB - 1) / DS_TB;
  stage(0);
  for (int blk = 0; blk < blocks; ++blk) {
    const int buf = blk & 1, t0 = blk * DS_TB, cnt = min(DS_TB, n - t0);
    if (blk + 1 < blocks) {
      stage(blk + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* kb = k_s + buf * DS_TB * DP;
    const float* qb = q_s + buf * DS_TB * DP;
    const float* gb = g_s + buf * DS_TB * 2;
    for (int t = warp; t < DS_TB; t += DS_THREADS / 32) {
      float a = 0.f;
      for (int d = lane; d < DP; d += 32) a = fmaf(kb[t * DP + d], qb[t * DP + d], a);
      a = warp_reduce_sum(a);
      if (lane == 0) {
        kq_s[t] = a;
        dec_s[t] = expf(gb[2 * t + 1]);
      }
    }
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {
      float kv[NR], sk = 0.f, sq = 0.f;
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const float4 k4 = *reinterpret_cast<const float4*>(kb + t * DP + 4 * (r + 8 * i));
        const float4 q4 = *reinterpret_cast<const float4*>(qb + t * DP + 4 * (r + 8 * i));
        kv[4 * i] = k4.x; kv[4 * i + 1] = k4.y; kv[4 * i + 2] = k4.z; kv[4 * i + 3] = k4.w;
        sk = fmaf(S[4 * i], k4.x, sk);
        sq = fmaf(S[4 * i], q4.x, sq);
        sk = fmaf(S[4 * i + 1], k4.y, sk);
        sq = fmaf(S[4 * i + 1], q4.y, sq);
        sk = fmaf(S[4 * i + 2], k4.z, sk);
        sq = fmaf(S[4 * i + 2], q4.z, sq);
        sk = fmaf(S[4 * i + 3], k4.w, sk);
        sq = fmaf(S[4 * i + 3], q4.w, sq);
      }
      sk = sum8(sk);
      sq = sum8(sq);
      const float g = dec_s[t];
      const float u = gb[2 * t] * (v_s[(buf * DS_TB + t) * DS_VB + col] - g * sk);
      if (r == 0) o_s[t * DS_VB + col] = g * sq + kq_s[t] * u;
#pragma unroll
      for (int i = 0; i < NR; ++i) S[i] = fmaf(kv[i], u, g * S[i]);
    }
    __syncthreads();
    T* out = static_cast<T*>(p.out) + (long long)(first + t0) * p.out_stride + (long long)h * p.V + v0;
    for (int i = tid; i < cnt * DS_VB; i += DS_THREADS) {
      const int t = i / DS_VB, c = i % DS_VB;
      if (v0 + c < p.V) out[(long long)t * p.out_stride + c] = dl_t<T>(o_s[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = 4 * (r + 8 * (i >> 2)) + (i & 3);
    if (col_on && row < p.D) st[row] = S[i];
  }
  // the last convolution inputs: the channels are dealt out over the CTAs of the sequence
  const T* proj = static_cast<const T*>(p.proj) + (long long)first * p.stride;
  T* ring = static_cast<T*>(p.ring) + (long long)slot * p.taps * C;
  const int parts = gridDim.x * gridDim.y, part = blockIdx.y * gridDim.x + blockIdx.x;
  for (int c = part * DS_THREADS + tid; c < C; c += parts * DS_THREADS)
    for (int t = max(0, n - p.taps); t < n; ++t)
      ring[(long long)((start + t) % p.taps) * C + c] = proj[(long long)t * p.stride + c];
}

// ---------------------------------------------------------------------------------------------------------------
// out = rmsnorm(out) * w * silu(gate) per (token, head), in place. One warp each.
template <typename T>
__global__ void __launch_bounds__(128) gated_norm_kernel(const DeltaParams p, int T_) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long i = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (i >= (long long)T_ * p.H) return;
  const long long t = i / p.H;
  const int h = (int)(i % p.H);
  T* o = static_cast<T*>(p.out) + t * p.out_stride + (long long)h * p.V;
  const T* gate = static_cast<const T*>(p.proj) + t * p.stride + 2 * p.Hk * p.D + p.H * p.V + (long long)h * p.V;
  const T* w = static_cast<const T*>(p.norm_w);
  float ss = 0.f;
  for (int c = lane; c < p.V; c += 32) {
    const float x = dl_f<T>(o[c]);
    ss += x * x;
  }
  const float inv = 1.f / sqrtf(warp_reduce_sum(ss) / (float)p.V + p.eps);
  for (int c = lane; c < p.V; c += 32) o[c] = dl_t<T>(dl_f<T>(o[c]) * inv * dl_f<T>(w[c]) * silu_f(dl_f<T>(gate[c])));
}

// ---------------------------------------------------------------------------------------------------------------
// Decode: one token per sequence, one CTA per (head, sequence), everything fused. The state columns are loaded before
// the convolution so that the memory traffic is in flight while the small work runs.
constexpr int DD_THREADS = 256, DD_NP = 4;
template <typename T, int NR>
__global__ void __launch_bounds__(DD_THREADS) delta_step_kernel(const DeltaParams p) {
  constexpr int DP = NR * 8;
  extern __shared__ float sm[];
  float* q_s = sm;          // [DP]
  float* k_s = q_s + DP;    // [DP]
  float* v_s = k_s + DP;    // [V]
  float* o_s = v_s + p.V;   // [V]
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane & 7, cw = warp * 4 + (lane >> 3);
  const int slot = p.slots[b], pos = p.seq_lens[b] - 1, group = p.H / p.Hk, hk = h / group;
  T* out = static_cast<T*>(p.out) + (long long)b * p.out_stride + (long long)h * p.V;
  if (slot < 0) {
    for (int c = tid; c < p.V; c += DD_THREADS) out[c] = dl_t<T>(0.f);
    return;
  }
  const int C = 2 * p.Hk * p.D + p.H * p.V;
  const T* proj = static_cast<const T*>(p.proj) + (long long)b * p.stride;
  float* st = p.state + ((long long)slot * p.H + h) * p.V * p.D;
  const bool vec = (p.D & 3) == 0;
  auto load_cols = [&](int cbase, float (&S)[DD_NP][NR]) {
#pragma unroll
    for (int j = 0; j < DD_NP; ++j) {
      const int col = cbase + j * 32 + cw;
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const int row = 4 * (r + 8 * i);
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (pos > 0 && col < p.V && row < p.D) {
          const float* src = st + (long long)col * p.D + row;
          if (vec) {
            x = __ldcs(reinterpret_cast<const float4*>(src));
          } else {
            x.x = src[0];
            if (row + 1 < p.D) x.y = src[1];
            if (row + 2 < p.D) x.z = src[2];
            if (row + 3 < p.D) x.w = src[3];
          }
        }
        S[j][4 * i] = x.x; S[j][4 * i + 1] = x.y; S[j][4 * i + 2] = x.z; S[j][4 * i + 3] = x.w;
      }
    }
  };
  float S[DD_NP][NR];
  load_cols(0, S);
  // convolution + silu of this head's channels
  T* ring = static_cast<T*>(p.ring) + (long long)slot * p.taps * C;
  const T* conv_w = static_cast<const T*>(p.conv_w);
  for (int i = tid; i < 2 * DP + p.V; i += DD_THREADS) {
    int c = -1;
    if (i < DP) c = i < p.D ? hk * p.D + i : -1;
    else if (i < 2 * DP) c = i - DP < p.D ? (p.Hk + hk) * p.D + i - DP : -1;
    else c = 2 * p.Hk * p.D + h * p.V + i - 2 * DP;
    float a = 0.f;
    if (c >= 0) {
      const T x = proj[c];
      const T* w = conv_w + (long long)c * p.taps;
      for (int j = p.taps - 1; j > 0; --j)
        if (pos - j >= 0) a = fmaf(dl_f<T>(w[p.taps - 1 - j]), dl_f<T>(ring[(long long)((pos - j) % p.taps) * C + c]), a);
      a = silu_f(fmaf(dl_f<T>(w[p.taps - 1]), dl_f<T>(x), a));
      if (i >= 2 * DP || h % group == 0) ring[(long long)(pos % p.taps) * C + c] = x;
    }
    sm[i] = a;
  }
  __syncthreads();
  if (warp < 2) {  // unit norms
    float* x = warp == 0 ? q_s : k_s;
    float ss = 0.f;
    for (int d = lane; d < DP; d += 32) ss += x[d] * x[d];
    const float mul = (warp == 0 ? 1.f / sqrtf((float)p.D) : 1.f) / sqrtf(warp_reduce_sum(ss) + UNIT_EPS);
    for (int d = lane; d < DP; d += 32) x[d] *= mul;
  }
  __syncthreads();
  const T* ba = proj + C + p.H * p.V;
  const float beta = sigmoid_f(dl_f<T>(ba[h]));
  const float g = expf(-expf(p.a_log[h]) * softplus_f(dl_f<T>(ba[p.H + h]) + p.dt_bias[h]));
  float kv[NR], qv[NR], kq = 0.f;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = 4 * (r + 8 * (i >> 2)) + (i & 3);
    kv[i] = k_s[row];
    qv[i] = q_s[row];
    kq = fmaf(kv[i], qv[i], kq);
  }
  kq = sum8(kq);
  for (int cbase = 0; cbase < p.V; cbase += DD_NP * 32) {
    if (cbase > 0) load_cols(cbase, S);
#pragma unroll
    for (int j = 0; j < DD_NP; ++j) {
      const int col = cbase + j * 32 + cw;
      float sk = 0.f, sq = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        sk = fmaf(S[j][i], kv[i], sk);
        sq = fmaf(S[j][i], qv[i], sq);
      }
      sk = sum8(sk);
      sq = sum8(sq);
      if (col < p.V) {
        const float u = beta * (v_s[col] - g * sk);
        if (r == 0) o_s[col] = g * sq + kq * u;
#pragma unroll
        for (int i = 0; i < NR / 4; ++i) {
          const int row = 4 * (r + 8 * i);
          if (row < p.D) {
            float4 x;
            x.x = fmaf(kv[4 * i], u, g * S[j][4 * i]);
            x.y = fmaf(kv[4 * i + 1], u, g * S[j][4 * i + 1]);
            x.z = fmaf(kv[4 * i + 2], u, g * S[j][4 * i + 2]);
            x.w = fmaf(kv[4 * i + 3], u, g * S[j][4 * i + 3]);
            float* dst = st + (long long)col * p.D + row;
            if (vec) {
              __stcs(reinterpret_cast<float4*>(dst), x);
            } else {
              dst[0] = x.x;
              if (row + 1 < p.D) dst[1] = x.y;
              if (row + 2 < p.D) dst[2] = x.z;
              if (row + 3 < p.D) dst[3] = x.w;
            }
          }
        }
      }
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = lane; c < p.V; c += 32) ss += o_s[c] * o_s[c];
  const float inv = 1.f / sqrtf(warp_reduce_sum(ss) / (float)p.V + p.eps);
  const T* gate = proj + C + (long long)h * p.V;
  const T* w = static_cast<const T*>(p.norm_w);
  for (int c = tid; c < p.V; c += DD_THREADS) out[c] = dl_t<T>(o_s[c] * inv * dl_f<T>(w[c]) * silu_f(dl_f<T>(gate[c])));
}

template <typename T>
static int run_prep(const DeltaParams& p, int max_q, cudaStream_t stream) {
  const dim3 g((max_q + DP_TT - 1) / DP_TT, (2 * p.Hk + p.H + 1 + 3) / 4, p.B), b(128);
  const int cpl = ((p.D > p.V ? p.D : p.V) + 31) / 32;
  cudaError_t e = cudaErrorInvalidValue;
#define VB_PREP(TAPS)                                                                                      \
  (cpl <= 1   ? vb_launch_pdl(delta_prep_kernel<T, TAPS, 1>, g, b, 0, stream, 1, p)                        \
   : cpl <= 2 ? vb_launch_pdl(delta_prep_kernel<T, TAPS, 2>, g, b, 0, stream, 1, p)                        \
   : cpl <= 4 ? vb_launch_pdl(delta_prep_kernel<T, TAPS, 4>, g, b, 0, stream, 1, p)                        \
              : vb_launch_pdl(delta_prep_kernel<T, TAPS, 8>, g, b, 0, stream, 1, p))
  e = p.taps <= 4 ? VB_PREP(4) : VB_PREP(8);
#undef VB_PREP
  vb_count_launch();
  return (int)e;
}

template <typename T, int NR>
static int run_scan(const DeltaParams& p, cudaStream_t stream) {
  constexpr int DP = NR * 8;
  const size_t smem = (4 * DS_TB * DP + 2 * DS_TB * DS_VB + 4 * DS_TB + 2 * DS_TB + DS_TB * DS_VB) * sizeof(float);
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(delta_scan_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr = true;
  }
  const dim3 g(p.H, (p.V + DS_VB - 1) / DS_VB, p.B);
  cudaError_t e = vb_launch_pdl(delta_scan_kernel<T, NR>, g, dim3(DS_THREADS), smem, stream, 1, p);
  vb_count_launch();
  return (int)e;
}

template <typename T, int NR>
static int run_step(const DeltaParams& p, cudaStream_t stream) {
  const size_t smem = (2 * NR * 8 + 2 * p.V) * sizeof(float);
  cudaError_t e = vb_launch_pdl(delta_step_kernel<T, NR>, dim3(p.H, p.B), dim3(DD_THREADS), smem, stream, 1, p);
  vb_count_launch();
  return (int)e;
}

template <typename T>
static int run_delta(const DeltaParams& p, int tokens, int max_q, cudaStream_t stream) {
  const int nr = p.D <= 32 ? 4 : p.D <= 64 ? 8 : p.D <= 128 ? 16 : 32;
  if (max_q == 1) {
    if (nr == 4) return run_step<T, 4>(p, stream);
    if (nr == 8) return run_step<T, 8>(p, stream);
    if (nr == 16) return run_step<T, 16>(p, stream);
    return run_step<T, 32>(p, stream);
  }
  int rc = run_prep<T>(p, max_q, stream);
  if (rc) return rc;
  rc = nr == 4 ? run_scan<T, 4>(p, stream) : nr == 8 ? run_scan<T, 8>(p, stream) : nr == 16 ? run_scan<T, 16>(p, stream)
                                                                                           : run_scan<T, 32>(p, stream);
  if (rc) return rc;
  const long long warps = (long long)tokens * p.H;
  cudaError_t e = vb_launch_pdl(gated_norm_kernel<T>, dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, stream, 1, p, tokens);
  vb_count_launch();
  return (int)e;
}

}  // namespace vb

using namespace vb;

// Limits: D, V <= 256, taps <= 8. max_q == 1 (every sequence brings exactly one token) takes the fused step and does not
// touch qkv / gates; otherwise qkv is fp32 scratch [T, 2 Hk D + H V] and gates fp32 scratch [T, 2 H].
extern "C" int vb_delta_rule(const void* proj, long long stride, const void* conv_w, const float* a_log,
                             const float* dt_bias, const void* norm_w, void* ring, float* state, const int* cu_q,
                             const int* seq_lens, const int* slots, float* qkv, float* gates, void* out,
                             long long out_stride, int T, int B, int max_q, int H, int Hk, int D, int V, int taps, float eps,
                             int f32, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_q <= 0) return 0;
  if (Hk <= 0 || H % Hk != 0 || D <= 0 || D > 256 || V <= 0 || V > 256 || taps < 1 || taps > 8 || B > 65535) return -3;
  if (max_q > 1 && (qkv == nullptr || gates == nullptr)) return -3;
  DeltaParams p{proj, stride, conv_w, a_log, dt_bias, norm_w, ring, state, cu_q, seq_lens, slots, qkv, gates, out,
                out_stride, B, H, Hk, D, V, taps, eps};
  const int rc = f32 ? run_delta<float>(p, T, max_q, stream) : run_delta<__nv_bfloat16>(p, T, max_q, stream);
  return rc ? rc : (int)cudaGetLastError();
}
