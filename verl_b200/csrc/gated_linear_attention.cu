// Gated linear attention over ragged batches with carried state (mixer of layer-list decoders).
//
// Per head with state S [D, V], decays a_t [D] (one per key channel), scaled q and plain k, v:
//     S <- diag(a_t) S + k_t v_t^T;   o_t = S^T q_t
// and the head's output is rmsnorm(o) * w * silu(gate). The decays come from a few numbers r per token that all heads share:
//     z = W r + b,   a = sigmoid(z)^(1 / tau)
//
// Input row of a token (one projection GEMM): [q (H D) | k (H D) | v (H V) | gate (H V) | r (rank) | ...].
// State of a sequence (slot s): fp32 state[s][H][V][D] (a column of S is contiguous). A sequence whose first token has position
// 0 starts from zero state whatever its slot holds; slot < 0 marks a padding row.
//
// Kernels:
//   gla_step    one token per sequence: everything fused (decode)
//   gla_chunk   chunks of up to 64 tokens on the tensor cores (bf16 serving), gated_norm behind it
//   gla_decay + gla_scan   token by token, state in registers, fp32 throughout (32-bit mode, sizes the chunks do not take)
#include "common.cuh"
#include "host_utils.h"
#include "state_ops.cuh"

namespace vb {

struct GlaParams {
  const void* proj;       // [T, stride]
  long long stride;
  const void* decay_w;    // [H D, rank]
  const float* decay_b;   // [H D]
  const void* norm_w;     // [V]
  float* state;           // [slots, H, V, D]
  const int* cu_q;        // [B + 1]
  const int* seq_lens;    // [B] tokens of the sequence up to and including this step's
  const int* slots;       // [B]
  float* decay;           // [T, H D] fp32 (scan path)
  void* out;              // [T, out_stride]
  long long out_stride;
  int H, D, V, rank, b0;  // b0: first sequence of a launch
  float inv_tau, eps;
};

// log(sigmoid(z))
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// z of channel c from the token's numbers r (shared memory or global)
template <typename T, typename R>
__device__ __forceinline__ float decay_logit(const GlaParams& p, int c, const R* r) {
  const T* w = static_cast<const T*>(p.decay_w) + (long long)c * p.rank;
  float z = p.decay_b[c];
  if ((p.rank & 7) == 0) {
    for (int i = 0; i < p.rank; i += 8) {
      float f[8];
      load_n<T, 8>(w + i, f);
#pragma unroll
      for (int k = 0; k < 8; ++k) z = fmaf(f[k], dl_f<R>(r[i + k]), z);
    }
  } else {
    for (int i = 0; i < p.rank; ++i) z = fmaf(dl_f<T>(w[i]), dl_f<R>(r[i]), z);
  }
  return z;
}

// ---------------------------------------------------------------------------------------------------------------
// Decode: one CTA per (head, sequence). The state columns are loaded first, so that the memory traffic is in flight while the
// decays are computed. Eight lanes share a column; lane r holds rows 4 (r + 8 i) + e.
constexpr int GS_THREADS = 256, GS_NP = 4;
template <typename T, int NR>
__global__ void __launch_bounds__(GS_THREADS, NR <= 16 ? 2 : 1) gla_step_kernel(const GlaParams p) {
  constexpr int DP = NR * 8;
  extern __shared__ float sm[];
  float* q_s = sm;            // [DP]
  float* k_s = q_s + DP;      // [DP]
  float* a_s = k_s + DP;      // [DP]
  float* v_s = a_s + DP;      // [V]
  float* o_s = v_s + p.V;     // [V]
  float* r_s = o_s + p.V;     // [rank]
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, b = p.b0 + blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane & 7, cw = warp * 4 + (lane >> 3);
  const int slot = p.slots[b], pos = p.seq_lens[b] - 1, t = p.cu_q[b];
  T* out = static_cast<T*>(p.out) + (long long)t * p.out_stride + (long long)h * p.V;
  if (slot < 0) {
    for (int c = tid; c < p.V; c += GS_THREADS) out[c] = dl_t<T>(0.f);
    return;
  }
  const T* row = static_cast<const T*>(p.proj) + (long long)t * p.stride;
  float* st = p.state + ((long long)slot * p.H + h) * p.V * p.D;
  const bool vec = (p.D & 3) == 0;
  auto load_cols = [&](int cbase, float (&S)[GS_NP][NR]) {
#pragma unroll
    for (int j = 0; j < GS_NP; ++j) {
      const int col = cbase + j * 32 + cw;
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const int d = 4 * (r + 8 * i);
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (pos > 0 && col < p.V && d < p.D) {
          const float* src = st + (long long)col * p.D + d;
          if (vec) {
            x = __ldcs(reinterpret_cast<const float4*>(src));
          } else {
            x.x = src[0];
            if (d + 1 < p.D) x.y = src[1];
            if (d + 2 < p.D) x.z = src[2];
            if (d + 3 < p.D) x.w = src[3];
          }
        }
        S[j][4 * i] = x.x; S[j][4 * i + 1] = x.y; S[j][4 * i + 2] = x.z; S[j][4 * i + 3] = x.w;
      }
    }
  };
  float S[GS_NP][NR];
  load_cols(0, S);
  const int HD = p.H * p.D, HV = p.H * p.V;
  for (int i = tid; i < p.rank; i += GS_THREADS) r_s[i] = dl_f<T>(row[2 * (HD + HV) + i]);
  const float qscale = 1.f / sqrtf((float)p.D);
  for (int d = tid; d < DP; d += GS_THREADS) {
    const bool on = d < p.D;
    q_s[d] = on ? dl_f<T>(row[h * p.D + d]) * qscale : 0.f;
    k_s[d] = on ? dl_f<T>(row[HD + h * p.D + d]) : 0.f;
  }
  for (int c = tid; c < p.V; c += GS_THREADS) v_s[c] = dl_f<T>(row[2 * HD + h * p.V + c]);
  __syncthreads();
  for (int d = tid; d < DP; d += GS_THREADS)
    a_s[d] = d < p.D ? expf(log_sigmoid(decay_logit<T>(p, h * p.D + d, r_s)) * p.inv_tau) : 0.f;
  __syncthreads();
  for (int cbase = 0; cbase < p.V; cbase += GS_NP * 32) {
    if (cbase > 0) load_cols(cbase, S);
    float v[GS_NP], o[GS_NP];
#pragma unroll
    for (int j = 0; j < GS_NP; ++j) {
      const int col = cbase + j * 32 + cw;
      v[j] = col < p.V ? v_s[col] : 0.f;
      o[j] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < NR / 4; ++i) {
      const int d = 4 * (r + 8 * i);
      const float4 q = *reinterpret_cast<const float4*>(q_s + d), k = *reinterpret_cast<const float4*>(k_s + d),
                   a = *reinterpret_cast<const float4*>(a_s + d);
#pragma unroll
      for (int j = 0; j < GS_NP; ++j) {
        float4 x = make_float4(S[j][4 * i], S[j][4 * i + 1], S[j][4 * i + 2], S[j][4 * i + 3]);
        x.x = fmaf(k.x, v[j], a.x * x.x);
        x.y = fmaf(k.y, v[j], a.y * x.y);
        x.z = fmaf(k.z, v[j], a.z * x.z);
        x.w = fmaf(k.w, v[j], a.w * x.w);
        o[j] = fmaf(x.x, q.x, fmaf(x.y, q.y, fmaf(x.z, q.z, fmaf(x.w, q.w, o[j]))));
        const int col = cbase + j * 32 + cw;
        if (col < p.V && d < p.D) {
          float* dst = st + (long long)col * p.D + d;
          if (vec) {
            __stcs(reinterpret_cast<float4*>(dst), x);
          } else {
            dst[0] = x.x;
            if (d + 1 < p.D) dst[1] = x.y;
            if (d + 2 < p.D) dst[2] = x.z;
            if (d + 3 < p.D) dst[3] = x.w;
          }
        }
      }
    }
#pragma unroll
    for (int j = 0; j < GS_NP; ++j) {
      const float x = sum8(o[j]);
      const int col = cbase + j * 32 + cw;
      if (r == 0 && col < p.V) o_s[col] = x;
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = lane; c < p.V; c += 32) ss += o_s[c] * o_s[c];
  const float inv = 1.f / sqrtf(warp_reduce_sum(ss) / (float)p.V + p.eps);
  const T* gate = row + 2 * HD + HV + (long long)h * p.V;
  const T* w = static_cast<const T*>(p.norm_w);
  for (int c = tid; c < p.V; c += GS_THREADS) out[c] = dl_t<T>(o_s[c] * inv * dl_f<T>(w[c]) * silu_f(dl_f<T>(gate[c])));
}

// ---------------------------------------------------------------------------------------------------------------
// decay[t][c] = sigmoid(z)^(1 / tau). One CTA per (token, 128 channels).
template <typename T>
__global__ void __launch_bounds__(128) gla_decay_kernel(const GlaParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.y * 128 + threadIdx.x, HD = p.H * p.D;
  const long long t = blockIdx.x;
  if (c >= HD) return;
  const T* r = static_cast<const T*>(p.proj) + t * p.stride + 2 * (HD + p.H * p.V);
  p.decay[t * HD + c] = expf(log_sigmoid(decay_logit<T>(p, c, r)) * p.inv_tau);
}

// One CTA per (head, 32 state columns, sequence); the lanes of a column as above. Tokens come in blocks through shared memory.
constexpr int GC_VB = 32, GC_TB = 16;
template <typename T, int NR>
__global__ void __launch_bounds__(GS_THREADS) gla_scan_kernel(const GlaParams p) {
  constexpr int DP = NR * 8;
  extern __shared__ float sm[];
  float* q_s = sm;                       // [TB][DP]
  float* k_s = q_s + GC_TB * DP;         // [TB][DP]
  float* a_s = k_s + GC_TB * DP;         // [TB][DP]
  float* v_s = a_s + GC_TB * DP;         // [TB][VB]
  float* o_s = v_s + GC_TB * GC_VB;      // [TB][VB]
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, v0 = blockIdx.y * GC_VB, b = p.b0 + blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane & 7, col = warp * 4 + (lane >> 3);
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;
  const int start = p.seq_lens[b] - n, HD = p.H * p.D;
  const bool col_on = v0 + col < p.V;
  float* st = p.state + (((long long)slot * p.H + h) * p.V + v0 + col) * p.D;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = 4 * (r + 8 * (i >> 2)) + (i & 3);
    S[i] = (start > 0 && col_on && d < p.D) ? st[d] : 0.f;
  }
  const T* proj = static_cast<const T*>(p.proj) + (long long)first * p.stride;
  const float* decay = p.decay + (long long)first * HD;
  const float qscale = 1.f / sqrtf((float)p.D);
  for (int t0 = 0; t0 < n; t0 += GC_TB) {
    const int cnt = min(GC_TB, n - t0);
    for (int i = tid; i < GC_TB * DP; i += GS_THREADS) {
      const int t = i / DP, d = i % DP;
      const bool on = t < cnt && d < p.D;
      const T* row = proj + (long long)(t0 + t) * p.stride + h * p.D + d;
      q_s[i] = on ? dl_f<T>(row[0]) * qscale : 0.f;
      k_s[i] = on ? dl_f<T>(row[HD]) : 0.f;
      a_s[i] = on ? decay[(long long)(t0 + t) * HD + h * p.D + d] : 0.f;
    }
    for (int i = tid; i < GC_TB * GC_VB; i += GS_THREADS) {
      const int t = i / GC_VB, c = i % GC_VB;
      v_s[i] = t < cnt && v0 + c < p.V ? dl_f<T>(proj[(long long)(t0 + t) * p.stride + 2 * HD + h * p.V + v0 + c]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {
      const float v = v_s[t * GC_VB + col];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const int at = t * DP + 4 * (r + 8 * i);
        const float4 q4 = *reinterpret_cast<const float4*>(q_s + at), k4 = *reinterpret_cast<const float4*>(k_s + at),
                     a4 = *reinterpret_cast<const float4*>(a_s + at);
        S[4 * i] = fmaf(k4.x, v, a4.x * S[4 * i]);
        S[4 * i + 1] = fmaf(k4.y, v, a4.y * S[4 * i + 1]);
        S[4 * i + 2] = fmaf(k4.z, v, a4.z * S[4 * i + 2]);
        S[4 * i + 3] = fmaf(k4.w, v, a4.w * S[4 * i + 3]);
        o = fmaf(S[4 * i], q4.x, o);
        o = fmaf(S[4 * i + 1], q4.y, o);
        o = fmaf(S[4 * i + 2], q4.z, o);
        o = fmaf(S[4 * i + 3], q4.w, o);
      }
      o = sum8(o);
      if (r == 0) o_s[t * GC_VB + col] = o;
    }
    __syncthreads();
    T* out = static_cast<T*>(p.out) + (long long)(first + t0) * p.out_stride + (long long)h * p.V + v0;
    for (int i = tid; i < cnt * GC_VB; i += GS_THREADS) {
      const int t = i / GC_VB, c = i % GC_VB;
      if (v0 + c < p.V) out[(long long)t * p.out_stride + c] = dl_t<T>(o_s[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = 4 * (r + 8 * (i >> 2)) + (i & 3);
    if (col_on && d < p.D) st[d] = S[i];
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Chunked form on the tensor cores. With b_t the running sum of log decays inside a chunk (per channel), S0 the state in front
// of it, Q~_t = q_t e^{b_t} and K~_s = k_s e^{-b_s}:
//     o_t = S0^T Q~_t + sum_{s<=t} (Q~_t . K~_s) v_s,      S = e^{b_last} (S0 + sum_s K~_s v_s^T)
// A chunk takes up to 64 tokens, fewer where a channel decays so far that e^{-b} would leave fp32's range: the walk then
// goes on behind the tokens it has taken, whatever their number.
//
// One CTA per (sequence, head, 128 state columns); tcgen05 with accumulators in TMEM (tokens = columns):
//     Z^T [d, t]      = W . r^T                                  (W in TMEM; the decays' logits)
//     P^T [s | s, t]  = [K~ hi; K~ lo] . (Q~ hi + Q~ lo)^T       (two partial sums of each score, added by the last product)
//     S^T [v, d]     += V^T . (K~ hi + K~ lo)                    (fp32 state in TMEM, decayed when it is read)
//     O^T [v, t]      = S0^T hi . (Q~ hi + Q~ lo)^T + S0^T lo . Q~ hi^T   (S0^T in TMEM)
//     O^T [v, t]     += [V; V]^T . P hi + V^T . P lo             (P: causal part of the scores)
// Every fp32 operand enters as two bf16 terms, so that products carry about 16 bits of both operands and sums are fp32; v and the
// numbers r are bf16 activations.
// Warps 0..15 make Q~ and K~ of chunk after chunk (two of them in shared memory), warps 16..23 turn scores into P, decay the state
// and store the outputs, warp 24 issues the products (but Z, which warp 0 does), warp 25 fetches q and k. A warp reads the TMEM lanes
// 32 (w % 4) ..; those of a group that share them have equal parts of the columns. q, k, v and r arrive by TMA.
constexpr int GK_C = 64, GK_MAKERS = 512, GK_USERS = 256, GK_THREADS = GK_MAKERS + GK_USERS + 64;
constexpr int GK_BUF = 32768;                      // Q~ or K~ of a chunk: per 64 channels hi | lo, [64 tokens] x 128 bytes
constexpr int GK_Q_OFF = 0, GK_K_OFF = 2 * GK_BUF;
constexpr int GK_V_OFF = GK_K_OFF + 2 * GK_BUF;    // v [64 tokens][128], two column blocks
constexpr int GK_P_OFF = GK_V_OFF + 16384;         // P hi [128 s][64 t] | P lo [64 s][64 t]
constexpr int GK_R_OFF = GK_P_OFF + 24576;         // q | k as they are, column blocks of 64: [64 tokens] x 128 bytes
constexpr int GK_A_OFF = GK_R_OFF + 32768;         // r [64 tokens][64]
constexpr int GK_SUM_OFF = GK_A_OFF + 8192;        // log decays of 16 tokens, [4][128] fp32
constexpr int GK_DEC_OFF = GK_SUM_OFF + 2048;      // e^{b_last} [128] of four chunks
constexpr int GK_BAR_OFF = GK_DEC_OFF + 2048;
constexpr int GK_SMEM = GK_BAR_OFF + 256 + 1024;
constexpr uint32_t GK_SC = 0, GK_O = 64, GK_ST = 128, GK_Z = 256, GK_W = 320, GK_SH = 352, GK_SL = 416;  // TMEM columns
constexpr float GK_RANGE = 90.f;                   // log2 of the largest e^{-b}: a stronger decay of one token does not show in fp32

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Barrier of the threads that make Q~ and K~, which also and-reduces a predicate.
__device__ __forceinline__ bool gk_bar_and(bool pred) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 q, %1, 0;\n\tbarrier.red.and.pred p, 1, 512, q;\n\tselp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(r)
      : "r"((uint32_t)pred)
      : "memory");
  return r != 0;
}

// ND: channels with those that are zero, 64 or 128
template <int ND>
__global__ void __launch_bounds__(GK_THREADS, 1)
gla_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                 const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmR, const GlaParams p, int* status) {
  extern __shared__ uint8_t smb[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smb) + 1023) & ~uintptr_t(1023));
  // Arrivals: by a copy (in), by the products (done), by the warps of a group. Barriers in pairs belong to chunks in turn.
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + GK_BAR_OFF);
  uint64_t *r_in = bars, *qk_in = bars + 1, *v_in = bars + 2, *z_done = bars + 3, *sc_done = bars + 4, *s_done = bars + 5,
           *o_done = bars + 7;                                                    // s_done: state and O of the state
  uint64_t *qk_made = bars + 9, *p_made = bars + 11, *s_made = bars + 12, *o_read = bars + 13;
  constexpr int NBAR = 14;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + NBAR);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* far = reinterpret_cast<int*>(tmem_slot + 2);
  int* cnt_s = reinterpret_cast<int*>(tmem_slot + 4);  // [4] tokens of a chunk
  float* sum_s = reinterpret_cast<float*>(smem + GK_SUM_OFF);
  pdl_wait();
  const int v0 = blockIdx.x * 128, h = blockIdx.y, b = p.b0 + blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, quad = warp & 3;
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;  // uniform for the CTA, before any barrier or allocation
  const int start = p.seq_lens[b] - n;
  const int VC = min(128, p.V - v0);             // columns of this CTA

  if (tid == 0) {
    for (int i = 0; i < NBAR; ++i) mbar_init(&bars[i], i < 9 ? 1 : i < 11 ? GK_MAKERS / 32 : GK_USERS / 32);
    *abort_flag = 0;
    *far = 0;
    mbar_fence_init();
  }
  if (warp == 24) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot, my = tmem + ((uint32_t)(quad * 32) << 16);
  pdl_trigger();  // TMEM is held
  const int row = quad * 32 + lane;              // TMEM lane: channel d, state column v or token s
  auto wait = [&](uint64_t* bar, uint32_t parity, int detail) {
    if (!*abort_flag && mbar_wait(bar, parity)) return true;
    report_error(status, ERR_WAIT_TMEM_FULL, detail);
    *abort_flag = 1;
    return false;
  };
  // what a warp has written to shared memory and read from TMEM is done: tell the barrier
  auto arrive = [&](uint64_t* bar) {
    fence_proxy_async_smem();
    tc_fence_before();
    __syncwarp();
    if (lane == 0) mbar_arrive(bar);
  };

  if (warp < 16) {
    // ----------------------------- Q~ and K~ (thread = channel, 16 tokens) -----------------------------
    const int grp = warp >> 2;
    const bool d_on = row < p.D;
    constexpr float LOG2E = 1.4426950408889634f;
    const float bias = d_on ? p.decay_b[h * p.D + row] * LOG2E : 0.f;
    const float qscale = 1.f / sqrtf((float)p.D);
    const int r_steps = (p.rank + 15) / 16;
    int loads_r = 0;
    auto load_r = [&](int t0) {
      mbar_arrive_expect_tx(r_in, 8192);
      tma_load_2d(smem + GK_A_OFF, &tmR, r_in, 0, first + t0);
      ++loads_r;
    };
    if (warp == 0) {
      if (elect_one()) {
        tma_prefetch_desc(&tmR);
        load_r(0);
      }
      __syncwarp();
    }
    if (grp == 0) {  // this channel's row of W
      uint32_t w[32];
      const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.decay_w) + (long long)(h * p.D + (d_on ? row : 0)) * p.rank;
#pragma unroll
      for (int i = 0; i < 32; ++i)
        w[i] = pack_bf16x2(d_on && 2 * i < p.rank ? dl_f(src[2 * i]) : 0.f, d_on && 2 * i + 1 < p.rank ? dl_f(src[2 * i + 1]) : 0.f);
      tmem_st_32x32(my + GK_W, w);
      tmem_st_wait();
    }
    constexpr uint32_t id_z = umma_idesc(1, 1, 0, 0, 128, 64);
    const uint64_t da = umma_smem_desc(smem_u32(smem) + GK_A_OFF, 16, 1024);
    bool ok = true;
    int t0 = 0;
    for (int c = 0; t0 < n; ++c) {
      tc_fence_before();
      ok = gk_bar_and(ok);  // everyone has read Z of the chunk before
      if (!ok) break;
      if (warp == 0) {
        if (elect_one()) {
          if (wait(r_in, c & 1, t0)) {
            tc_fence_after();
            for (int k = 0; k < r_steps; ++k) tc_mma_f16_ta(tmem + GK_Z, tmem + GK_W + k * 8, da + k * 2, id_z, k != 0);
            tc_commit(z_done);
          }
        }
        __syncwarp();
      }
      // running log2 decays of this thread's channel over its tokens
      float lb[16];
      ok = wait(z_done, c & 1, t0 + 1);
      tc_fence_after();
      {
        uint32_t z[16];
        tmem_ld_32x16(my + GK_Z + grp * 16, z);
        tmem_ld_wait();
        const int in = d_on ? n - t0 - grp * 16 : 0;
        float run = 0.f;
#pragma unroll
        for (int i = 0; i < 16; ++i) {  // log2 sigmoid(z) = min(z', 0) - log2(1 + 2^-|z'|), z' = z log2(e)
          const float y = fmaf(__uint_as_float(z[i]), LOG2E, bias);
          const float l = (fminf(y, 0.f) - lg2(1.f + ex2(-fabsf(y)))) * p.inv_tau;
          run += i < in ? l : 0.f;
          lb[i] = run;
        }
        sum_s[grp * 128 + row] = run;
      }
      gk_bar_and(true);
      {
        float before = 0.f;
#pragma unroll
        for (int g = 0; g < 3; ++g)
          if (g < grp) before += sum_s[g * 128 + row];
#pragma unroll
        for (int i = 0; i < 16; ++i) lb[i] += before;
      }
      int cnt = min(GK_C, n - t0);  // tokens of this chunk
      if (!gk_bar_and(lb[15] >= -GK_RANGE)) {  // the largest power of two of them that stays within the range
        int out = 0;
#pragma unroll
        for (int k = 0; k < 6; ++k) {
          const int t = (1 << k) - 1;
          if ((t >> 4) == grp && lb[t & 15] < -GK_RANGE) out |= 1 << k;
        }
        if (out) atomicOr(far, out);
        gk_bar_and(true);
        out = *far;
        int m = 1;
        while (m < 32 && !(out & (2 * m))) m *= 2;
        cnt = min(cnt, m);
#pragma unroll
        for (int i = 0; i < 16; ++i) lb[i] = fmaxf(lb[i], -GK_RANGE);
        gk_bar_and(true);
        if (tid == 0) *far = 0;
      }
      const int t1 = t0 + cnt, buf = c & 1;
      if (warp == 0) {
        if (elect_one() && t1 < n) load_r(t1);
        __syncwarp();
      }
      // everyone is through with chunk c - 2 (O is the last that is made of it)
      if (c > 1) ok = wait(&o_done[buf], ((c >> 1) + 1) & 1, t0 + 2) && ok;
      ok = wait(qk_in, c & 1, t0 + 3) && ok;
      // lanes in pairs, each lane two channels of eight tokens: the even one the first eight of the sixteen
      if (row < ND) {
        const bool odd = lane & 1;
        const int d = row & ~1, g = (d >> 3) & 7;
        float* dec = reinterpret_cast<float*>(smem + GK_DEC_OFF) + (c & 3) * 128 + d;
        uint8_t* dst = smem + buf * GK_BUF + (d >> 6) * 16384 + (d & 7) * 2;
        const uint8_t* src = smem + GK_R_OFF + (d >> 6) * 8192 + (d & 7) * 2;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float own = odd ? lb[8 + (j ^ 4)] : lb[j], give = odd ? lb[j] : lb[8 + (j ^ 4)];
          const float got = __shfl_xor_sync(0xffffffffu, give, 1);
          const float b0 = odd ? got : own, b1 = odd ? own : got;
          const int t = grp * 16 + (odd ? 8 + (j ^ 4) : j);
          const int at = t * 128 + ((g ^ (t & 7)) << 4);
          const uint32_t q2 = *reinterpret_cast<const uint32_t*>(src + at), k2 = *reinterpret_cast<const uint32_t*>(src + 16384 + at);
          const bool on = t < cnt;  // other tokens: zeros
          const float e0 = ex2(b0), e1 = ex2(b1), f0 = ex2(-b0), f1 = ex2(-b1), qs = on ? qscale : 0.f;
          if (t == cnt - 1) *reinterpret_cast<float2*>(dec) = make_float2(e0, e1);
          uint32_t qh, ql, kh, kl;
          split2(__uint_as_float(q2 << 16) * (qs * e0), __uint_as_float(q2 & 0xffff0000u) * (qs * e1), qh, ql);
          split2(__uint_as_float(k2 << 16) * (on ? f0 : 0.f), __uint_as_float(k2 & 0xffff0000u) * (on ? f1 : 0.f), kh, kl);
          *reinterpret_cast<uint32_t*>(dst + at + GK_Q_OFF) = qh;
          *reinterpret_cast<uint32_t*>(dst + at + GK_Q_OFF + 8192) = ql;
          *reinterpret_cast<uint32_t*>(dst + at + GK_K_OFF) = kh;
          *reinterpret_cast<uint32_t*>(dst + at + GK_K_OFF + 8192) = kl;
        }
      }
      if (tid == 0) cnt_s[c & 3] = cnt;
      arrive(&qk_made[buf]);
      t0 = t1;
    }
    // no copy is in flight when the CTA ends, whatever ended it
    if (loads_r > 0) mbar_wait(r_in, (loads_r - 1) & 1);
  } else if (warp < 24) {
    // ------------------------- P, the state, the outputs (every warp on its own) -------------------------
    const int half = (warp >> 2) & 1;
    int loads_v = 0;
    auto load_v = [&](int t0) {
      if (warp == 16) {
        if (elect_one()) {
          mbar_arrive_expect_tx(v_in, 16384);
          tma_load_3d(smem + GK_V_OFF, &tmV, v_in, v0, h, first + t0);
          tma_load_3d(smem + GK_V_OFF + 8192, &tmV, v_in, v0 + 64, h, first + t0);
          ++loads_v;
        }
        __syncwarp();
      }
    };
    load_v(0);
    float* st = p.state + (((long long)slot * p.H + h) * p.V + v0 + row) * p.D;
    constexpr int SR = ND / 64;  // this thread's channels of column v, 32 at a time
    // fp32 accumulator and two bf16 terms of 32 channels
    auto put_state = [&](int c0, const uint32_t (&x)[32]) {
      tmem_st_32x32(my + GK_ST + c0, x);
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        uint32_t y[16];
#pragma unroll
        for (int e = 0; e < 8; ++e)
          split2(__uint_as_float(x[16 * k + 2 * e]), __uint_as_float(x[16 * k + 2 * e + 1]), y[e], y[8 + e]);
        tmem_st_32x8(my + GK_SH + c0 / 2 + 8 * k, y);
        tmem_st_32x8(my + GK_SL + c0 / 2 + 8 * k, y + 8);
      }
    };
#pragma unroll
    for (int k = 0; k < SR; ++k) {
      const int c0 = (half * SR + k) * 32;
      uint32_t x[32];
#pragma unroll
      for (int e = 0; e < 32; ++e) x[e] = start > 0 && row < VC && c0 + e < p.D ? __float_as_uint(st[c0 + e]) : 0u;
      put_state(c0, x);
    }
    tmem_st_wait();
    arrive(s_made);
    int t0 = 0;
    for (int c = 0; t0 < n; ++c) {
      const int buf = c & 1;
      // scores: this thread's row s (hi or lo term of K~) and 32 tokens t
      if (!__all_sync(0xffffffffu, wait(&qk_made[buf], (c >> 1) & 1, t0 + 4) && wait(sc_done, c & 1, t0 + 5))) break;
      tc_fence_after();
      const int cnt = cnt_s[c & 3], t1 = t0 + cnt;
      {
        uint32_t x[32];
        tmem_ld_32x32(my + GK_SC + half * 32, x);
        tmem_ld_wait();
        const int s = row & 63;
        uint8_t* dst = smem + GK_P_OFF + row * 128;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int e = 8 * j + 2 * k, t = half * 32 + e;
            split2(t >= s ? __uint_as_float(x[e]) : 0.f, t + 1 >= s ? __uint_as_float(x[e + 1]) : 0.f, hi[k], lo[k]);
          }
          const int off = ((4 * half + j) ^ (row & 7)) << 4;
          *reinterpret_cast<uint4*>(dst + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          if (quad < 2) *reinterpret_cast<uint4*>(dst + 16384 + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      arrive(p_made);
      // the state behind the chunk
      if (!__all_sync(0xffffffffu, wait(&s_done[buf], (c >> 1) & 1, t0 + 6))) break;
      tc_fence_after();
      const float* dec = reinterpret_cast<const float*>(smem + GK_DEC_OFF) + (c & 3) * 128;
#pragma unroll
      for (int k = 0; k < SR; ++k) {
        const int c0 = (half * SR + k) * 32;
        uint32_t x[32];
        tmem_ld_32x32(my + GK_ST + c0, x);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e += 4) {
          const float4 d4 = *reinterpret_cast<const float4*>(dec + c0 + e);
          x[e] = __float_as_uint(__uint_as_float(x[e]) * d4.x);
          x[e + 1] = __float_as_uint(__uint_as_float(x[e + 1]) * d4.y);
          x[e + 2] = __float_as_uint(__uint_as_float(x[e + 2]) * d4.z);
          x[e + 3] = __float_as_uint(__uint_as_float(x[e + 3]) * d4.w);
        }
        if (t1 < n) {
          put_state(c0, x);
        } else if (row < VC) {
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if (c0 + e < p.D) st[c0 + e] = __uint_as_float(x[e]);
        }
      }
      tmem_st_wait();
      arrive(s_made);
      if (!__all_sync(0xffffffffu, wait(&o_done[buf], (c >> 1) & 1, t0 + 7))) break;
      tc_fence_after();
      if (t1 < n) load_v(t1);
      // outputs: lanes in pairs, two columns v of one token each
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (long long)(first + t0 + half * 32 + (lane & 1)) * p.out_stride +
                           (long long)h * p.V + v0 + (row & ~1);
      const int left = (row & ~1) < VC ? cnt - half * 32 - (lane & 1) : 0;
      uint32_t x[32];
      tmem_ld_32x32(my + GK_O + half * 32, x);
      tmem_ld_wait();
      arrive(o_read);
#pragma unroll
      for (int e = 0; e < 32; e += 2) {
        const bool odd = lane & 1;
        const float got = __shfl_xor_sync(0xffffffffu, __uint_as_float(odd ? x[e] : x[e + 1]), 1);
        const float own = __uint_as_float(odd ? x[e + 1] : x[e]);
        if (e < left) *reinterpret_cast<uint32_t*>(out) = odd ? pack_bf16x2(got, own) : pack_bf16x2(own, got);
        out += 2 * p.out_stride;
      }
      t0 = t1;
    }
    if (loads_v > 0) mbar_wait(v_in, (loads_v - 1) & 1);
  } else if (warp == 25) {
    // ----------------------------------- q and k -----------------------------------
    if (elect_one()) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      int t0 = 0, c = 0;
      for (; t0 < n; ++c) {
        mbar_arrive_expect_tx(qk_in, 2 * (ND / 64) * 8192);
#pragma unroll
        for (int x = 0; x < ND / 64; ++x) {
          tma_load_3d(smem + GK_R_OFF + x * 8192, &tmQ, qk_in, x * 64, h, first + t0);
          tma_load_3d(smem + GK_R_OFF + 16384 + x * 8192, &tmK, qk_in, x * 64, h, first + t0);
        }
        if (!wait(&qk_made[c & 1], (c >> 1) & 1, t0 + 13)) {
          mbar_wait(qk_in, c & 1);
          break;
        }
        t0 += cnt_s[c & 3];
      }
    }
  } else if (elect_one()) {
    // ---------------------------------- products ----------------------------------
    constexpr int K_STEPS = ND / 16;
    constexpr uint32_t id_kk = umma_idesc(1, 1, 0, 0, 128, 64);           // both K-major
    constexpr uint32_t id_mm = umma_idesc(1, 1, 1, 1, 128, 64);           // both MN-major
    constexpr uint32_t id_st = umma_idesc(1, 1, 1, 1, 128, ND);
    // a step of 32 bytes (K-major) or 2048 bytes (MN-major) adds to the address field of a descriptor
    const uint32_t base = smem_u32(smem);
    const uint64_t dq0 = umma_smem_desc(base + GK_Q_OFF, 16, 1024), dk0 = umma_smem_desc(base + GK_K_OFF, 16, 1024),
                   dkt0 = umma_smem_desc(base + GK_K_OFF, 16384, 1024), dv = umma_smem_desc(base + GK_V_OFF, 8192, 1024),
                   dp = umma_smem_desc(base + GK_P_OFF, 8192, 1024);
    int t0 = 0;
    for (int c = 0; t0 < n; ++c) {
      const int buf = c & 1;
      const uint64_t dq = dq0 + buf * (GK_BUF / 16), dk = dk0 + buf * (GK_BUF / 16), dkt = dkt0 + buf * (GK_BUF / 16);
      if (!wait(&qk_made[buf], (c >> 1) & 1, t0 + 8)) break;
      tc_fence_after();
#pragma unroll
      for (int term = 0; term < 2; ++term)
#pragma unroll
        for (int k = 0; k < K_STEPS; ++k)
          tc_mma_f16(tmem + GK_SC, dk + (k >> 2) * 1024 + (k & 3) * 2, dq + term * 512 + (k >> 2) * 1024 + (k & 3) * 2, id_kk,
                     term != 0 || k != 0);
      tc_commit(sc_done);
      if (!wait(v_in, c & 1, t0 + 9) || !wait(s_made, c & 1, t0 + 10)) break;
      tc_fence_after();
#pragma unroll
      for (int term = 0; term < 2; ++term)
#pragma unroll
        for (int k = 0; k < GK_C / 16; ++k)
          tc_mma_f16(tmem + GK_ST, dv + k * 128, dkt + term * 512 + k * 128, id_st, 1);
      if (c > 0 && !wait(o_read, (c - 1) & 1, t0 + 11)) break;
      tc_fence_after();
#pragma unroll
      for (int term = 0; term < 3; ++term)  // hi hi, hi lo, lo hi
#pragma unroll
        for (int k = 0; k < K_STEPS; ++k)
          tc_mma_f16_ta(tmem + GK_O, tmem + (term == 2 ? GK_SL : GK_SH) + k * 8,
                        dq + (term == 1 ? 512 : 0) + (k >> 2) * 1024 + (k & 3) * 2, id_kk, term != 0 || k != 0);
      tc_commit(&s_done[buf]);
      if (!wait(p_made, c & 1, t0 + 12)) break;
      tc_fence_after();
#pragma unroll
      for (int k = 0; k < 12; ++k)  // P hi of both partial sums, P lo of the first
        tc_mma_f16(tmem + GK_O, dv + (k & 3) * 128, dp + k * 128, id_mm, 1);
      tc_commit(&o_done[buf]);
      t0 += cnt_s[c & 3];
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 24) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// proj of T tokens; sequences from p.b0 on
static int run_gla_chunks(const GlaParams& p, int T, int sequences, int* status, cudaStream_t stream) {
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(gla_chunk_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, GK_SMEM));
    VB_CUDA_CHECK(cudaFuncSetAttribute(gla_chunk_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, GK_SMEM));
    attr = true;
  }
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(p.proj);
  const uint64_t D = p.D, H = p.H, V = p.V, row = (uint64_t)p.stride * 2;
  CUtensorMap tmQ, tmK, tmV, tmR;
  int rc = vb_make_tmap_3d(&tmQ, x, 2, D, H, T, D * 2, row, 64, 1, GK_C);
  if (!rc) rc = vb_make_tmap_3d(&tmK, x + H * D, 2, D, H, T, D * 2, row, 64, 1, GK_C);
  if (!rc) rc = vb_make_tmap_3d(&tmV, x + 2 * H * D, 2, V, H, T, V * 2, row, 64, 1, GK_C);
  if (!rc) rc = vb_make_tmap_2d(&tmR, x + 2 * H * (D + V), 2, p.rank, T, row, 64, GK_C);
  if (rc) return rc;
  const dim3 g((p.V + 127) / 128, p.H, sequences), blk(GK_THREADS);
  rc = (int)(p.D <= 64 ? vb_launch_pdl(gla_chunk_kernel<64>, g, blk, GK_SMEM, stream, 1, tmQ, tmK, tmV, tmR, p, status)
                       : vb_launch_pdl(gla_chunk_kernel<128>, g, blk, GK_SMEM, stream, 1, tmQ, tmK, tmV, tmR, p, status));
  vb_count_launch();
  return rc;
}

template <typename T, int NR>
static int run_gla_step(const GlaParams& p, int B, cudaStream_t stream) {
  const size_t smem = (3 * NR * 8 + 2 * p.V + p.rank) * sizeof(float);
  cudaError_t e = vb_launch_pdl(gla_step_kernel<T, NR>, dim3(p.H, B), dim3(GS_THREADS), smem, stream, 1, p);
  vb_count_launch();
  return (int)e;
}

template <typename T, int NR>
static int run_gla_scan(const GlaParams& p, int B, cudaStream_t stream) {
  const size_t smem = (3 * GC_TB * NR * 8 + 2 * GC_TB * GC_VB) * sizeof(float);
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(gla_scan_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr = true;
  }
  const dim3 g(p.H, (p.V + GC_VB - 1) / GC_VB, B);
  cudaError_t e = vb_launch_pdl(gla_scan_kernel<T, NR>, g, dim3(GS_THREADS), smem, stream, 1, p);
  vb_count_launch();
  return (int)e;
}

template <typename T>
static int run_gla(GlaParams p, int T_, int B, int singles, int chunk, int* status, cudaStream_t stream) {
  const int nr = p.D <= 32 ? 4 : p.D <= 64 ? 8 : p.D <= 128 ? 16 : 32;
  int rc = 0;
  if (singles > 0) {
    rc = nr == 4    ? run_gla_step<T, 4>(p, singles, stream)
         : nr == 8  ? run_gla_step<T, 8>(p, singles, stream)
         : nr == 16 ? run_gla_step<T, 16>(p, singles, stream)
                    : run_gla_step<T, 32>(p, singles, stream);
    if (rc || singles == B) return rc;
  }
  p.b0 = singles;
  if (chunk) {
    rc = run_gla_chunks(p, T_, B - singles, status, stream);
  } else {
    cudaError_t e = vb_launch_pdl(gla_decay_kernel<T>, dim3(T_, (p.H * p.D + 127) / 128), dim3(128), 0, stream, 1, p);
    vb_count_launch();
    if (e != cudaSuccess) return (int)e;
    rc = nr == 4    ? run_gla_scan<T, 4>(p, B - singles, stream)
         : nr == 8  ? run_gla_scan<T, 8>(p, B - singles, stream)
         : nr == 16 ? run_gla_scan<T, 16>(p, B - singles, stream)
                    : run_gla_scan<T, 32>(p, B - singles, stream);
  }
  if (rc) return rc;
  // the leading sequences have one token each, which the step has finished
  T* out = static_cast<T*>(p.out) + (long long)singles * p.out_stride;
  const T* gate = static_cast<const T*>(p.proj) + (long long)singles * p.stride + 2 * p.H * p.D + p.H * p.V;
  return launch_gated_norm<T>(out, p.out_stride, gate, p.stride, p.norm_w, p.H, p.V, p.eps, T_ - singles, stream);
}

}  // namespace vb

using namespace vb;

// 1 if the chunked form serves these sizes (bf16 only).
extern "C" int vb_gla_chunk_supported(int H, int D, int V, int rank) {
  return H > 0 && D >= 8 && D <= 128 && (D & 7) == 0 && V >= 8 && V <= 256 && (V & 7) == 0 && rank > 0 && rank <= 64;
}

// Limits: D, V <= 256, rank <= 4096. The leading `singles` sequences bring one token each (singles == B: all do); the others take the
// chunked form (chunk) or the scan, with decay fp32 scratch [T, H D].
extern "C" int vb_gla(const void* proj, long long stride, const void* decay_w, const float* decay_b, const void* norm_w,
                      float* state, const int* cu_q, const int* seq_lens, const int* slots, float* decay, void* out,
                      long long out_stride, int T, int B, int singles, int max_q, int H, int D, int V, int rank, float tau,
                      float eps, int f32, int chunk, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_q <= 0) return 0;
  if (H <= 0 || D <= 0 || D > 256 || V <= 0 || V > 256 || rank <= 0 || rank > 4096 || !(tau > 0.f) || singles < 0 || singles > B ||
      B > 65535 || H > 65535 ||
      (singles < B && (chunk ? !vb_gla_chunk_supported(H, D, V, rank) || f32 || (stride & 7) || (out_stride & 7) : decay == nullptr)))
    return -3;
  GlaParams p{proj, stride, decay_w, decay_b, norm_w, state, cu_q, seq_lens, slots, decay, out, out_stride, H, D, V, rank, 0,
              1.f / tau, eps};
  const int rc = f32 ? run_gla<float>(p, T, B, singles, chunk, status, stream)
                     : run_gla<__nv_bfloat16>(p, T, B, singles, chunk, status, stream);
  return rc ? rc : (int)cudaGetLastError();
}
