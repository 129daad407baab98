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
// Kernels:
//   delta_step   one token per sequence: everything fused (decode)
//   delta_prep   convolution, silu, unit norms, gates of every token, then either
//     delta_scan   token by token, state in registers, fp32 throughout (32-bit mode, short portions, any head size), or
//     delta_chunk_prep + delta_chunk_scan   chunks of 64 tokens on the tensor cores (bf16 serving)
//   gated_norm   the output norm and gate
//
// Chunked form. With G_t the running sum of log decays inside a chunk, S0 the state in front of it and u_t the write of
// token t, unrolling the recurrence gives
//     u_t = beta_t (v_t - e^{G_t} S0^T k_t - sum_{s<t} e^{G_t - G_s} (k_t . k_s) u_s)       i.e. (I + A) U = B (V - ...)
//     o_t = e^{G_t} S0^T q_t + sum_{s<=t} e^{G_t - G_s} (q_t . k_s) u_s
//     S   = e^{G_last} S0 + sum_s e^{G_last - G_s} k_s u_s^T
// delta_chunk_prep computes T = (I + A)^-1 B and, with P the matrix of the second sum, P T for all chunks in parallel;
// delta_chunk_scan walks a sequence's chunks on tcgen05 with S in fp32 accumulators. Precision: the convolved q and k are bf16
// activations and enter the products unnormalised, their fp32 unit-norm factors multiply the results; every other
// operand (S, T, P T, U and the right-hand side) is split into two bf16 terms, so that products carry about 16 bits of
// both operands and sums are fp32.
#include "common.cuh"
#include "host_utils.h"
#include "state_ops.cuh"

namespace vb {

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
  void* qkv;               // [T, C]: fp32, unit q and k (scan path); bf16, unnormalised (chunk path)
  float* unit;             // [T, 2 Hk] fp32 factors that make q (times D^-1/2) and k unit vectors (chunk path)
  float* gates;            // [T, 2 H] fp32: beta | log decay (scan path)
  void* out;               // [T, out_stride]
  long long out_stride;
  int B, H, Hk, D, V, taps;
  float eps;
};

// ---------------------------------------------------------------------------------------------------------------
// One warp per (sequence, tile of tokens, head row); lanes across the head's channels, a sliding window of inputs in
// registers. Head rows: Hk of q, Hk of k, H of v; a few more rows do the gates.
constexpr int DP_TT = 64;  // tokens per tile
constexpr int DP_GATE_ROWS = 8;  // warps that share a tile's gates
template <typename T, int TAPS, int CPL>
__global__ void __launch_bounds__(128, CPL * TAPS <= 16 ? 8 : 1) delta_prep_kernel(const DeltaParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, r = blockIdx.y * 4 + (threadIdx.x >> 5), b = blockIdx.z;
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first;
  const int t0 = blockIdx.x * DP_TT, t1 = min(n, t0 + DP_TT);
  const int slot = p.slots[b], rows = 2 * p.Hk + p.H;
  if (t0 >= n || r >= rows + DP_GATE_ROWS || slot < 0) return;
  const int start = p.seq_lens[b] - n;
  const int C = 2 * p.Hk * p.D + p.H * p.V;
  const T* proj = static_cast<const T*>(p.proj) + (long long)first * p.stride;
  if (r >= rows) {
#pragma unroll 4
    for (int i = (r - rows) * 32 + lane; i < (t1 - t0) * p.H; i += 32 * DP_GATE_ROWS) {
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
  // Lane l owns channels l * CPL .. of the head, loaded as one vector where sizes and strides allow.
  const bool vec = ((p.D | p.V | C | (int)p.stride) & (CPL - 1)) == 0;
  const int cl = lane * CPL;
  auto row_in = [&](const T* row, float (&x)[CPL]) {
    if (vec) {
      if (cl < size) {
        load_n<T, CPL>(row + cl, x);
      } else {
#pragma unroll
        for (int i = 0; i < CPL; ++i) x[i] = 0.f;
      }
    } else {
#pragma unroll
      for (int i = 0; i < CPL; ++i) x[i] = cl + i < size ? dl_f<T>(row[cl + i]) : 0.f;
    }
  };
  // w[j], hist[j]: tap and input of the token j places back; taps beyond p.taps stay zero
  float w[TAPS][CPL], hist[TAPS][CPL];
  float wv[CPL * TAPS];
  const bool wvec = vec && p.taps == TAPS;
  if (wvec && cl < size) load_n<T, CPL * TAPS>(cw + cl * TAPS, wv);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    const int t = t0 - j;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      w[j][i] = 0.f;
      if (cl + i < size && j < p.taps) w[j][i] = wvec ? wv[i * TAPS + TAPS - 1 - j] : dl_f<T>(cw[(cl + i) * p.taps + p.taps - 1 - j]);
      hist[j][i] = 0.f;
    }
    if (j > 0 && j < p.taps) {
      if (t >= 0) row_in(proj + (long long)t * p.stride + c0, hist[j]);
      else if (start + t >= 0) row_in(ring + (long long)((start + t) % p.taps) * C, hist[j]);
    }
  }
  const float qscale = r < p.Hk ? 1.f / sqrtf((float)p.D) : 1.f;
  constexpr int PRE = 4;  // tokens whose loads are in flight together
  const T* src = proj + (long long)t0 * p.stride + c0;
  for (int tb = t0; tb < t1; tb += PRE) {
    float xin[PRE][CPL];
#pragma unroll
    for (int k = 0; k < PRE; ++k, src += p.stride)
      if (tb + k < t1) row_in(src, xin[k]);
#pragma unroll
    for (int k = 0; k < PRE; ++k) {
      const int t = tb + k;
      if (t >= t1) break;
      float y[CPL], ss = 0.f;
#pragma unroll
      for (int i = 0; i < CPL; ++i) {
        hist[0][i] = xin[k][i];
        float a = 0.f;
#pragma unroll
        for (int j = TAPS - 1; j >= 0; --j) a = fmaf(w[j][i], hist[j][i], a);
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j) hist[j][i] = hist[j - 1][i];
        y[i] = silu_f(a);
        ss += y[i] * y[i];  // channels past the head give silu(0) = 0
      }
      float mul = 1.f;
      if (qk) mul = qscale * rsqrtf(warp_reduce_sum(ss) + UNIT_EPS);
      float* dst = static_cast<float*>(p.qkv) + (long long)(first + t) * C + c0 + cl;
#pragma unroll
      for (int i = 0; i < CPL; ++i) y[i] *= mul;
      if (vec) {
        if (cl < size) store_n<float, CPL>(dst, y);
      } else {
#pragma unroll
        for (int i = 0; i < CPL; ++i)
          if (cl + i < size) dst[i] = y[i];
      }
    }
  }
}

// The same for the chunked form, bf16: one CTA per (sequence, tile of tokens, 128 channels of one head row). The tile and
// the taps in front of it come into shared memory with all loads in flight; a warp takes 16 tokens, a lane 4 channels.
template <int TAPS>
__global__ void __launch_bounds__(128) delta_prep_tile_kernel(const DeltaParams p) {
  __shared__ __align__(16) __nv_bfloat16 x_s[DP_TT + TAPS - 1][128];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, b = blockIdx.z;
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, t0 = blockIdx.x * DP_TT, t1 = min(n, t0 + DP_TT);
  const int slot = p.slots[b];
  if (t0 >= n || slot < 0) return;
  const int start = p.seq_lens[b] - n, C = 2 * p.Hk * p.D + p.H * p.V, vb = (p.V + 127) / 128;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj) + (long long)first * p.stride;
  int r = blockIdx.y;
  if (r == 2 * p.Hk + p.H * vb) {  // the gates
    for (int i = tid; i < (t1 - t0) * p.H; i += 128) {
      const int t = t0 + i / p.H, h = i % p.H;
      const __nv_bfloat16* row = proj + (long long)t * p.stride + C + p.H * p.V;
      float* g = p.gates + (long long)(first + t) * 2 * p.H;
      g[h] = sigmoid_f(dl_f(row[h]));
      g[p.H + h] = -expf(p.a_log[h]) * softplus_f(dl_f(row[p.H + h]) + p.dt_bias[h]);
    }
    return;
  }
  const bool qk = r < 2 * p.Hk;
  const int rv = r - 2 * p.Hk;
  const int c0 = qk ? r * p.D : 2 * p.Hk * p.D + rv / vb * p.V + rv % vb * 128;
  const int size = qk ? p.D : min(128, p.V - rv % vb * 128);
  const __nv_bfloat16* ring = static_cast<const __nv_bfloat16*>(p.ring) + (long long)slot * p.taps * C + c0;
  for (int i = tid; i < (DP_TT + TAPS - 1) * 16; i += 128) {
    const int k = i >> 4, c = (i & 15) * 8, t = t0 + k - (TAPS - 1);  // row k holds token t
    const bool cur = t >= 0, past = !cur && start + t >= 0 && -t < p.taps;
    const bool on = c < size && t < t1 && (cur || past);
    const __nv_bfloat16* src = !on ? proj : cur ? proj + (long long)t * p.stride + c0 + c : ring + (long long)((start + t) % p.taps) * C + c;
    cp_async16(&x_s[k][c], src, on);
  }
  cp_async_commit();
  const int cl = lane * 4;
  float w[TAPS][4];  // w[j]: tap of the token j places back
  const __nv_bfloat16* cw = static_cast<const __nv_bfloat16*>(p.conv_w) + (long long)(c0 + cl) * p.taps;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j][i] = cl < size && j < p.taps ? dl_f(cw[i * p.taps + p.taps - 1 - j]) : 0.f;
  const float qscale = r < p.Hk ? 1.f / sqrtf((float)p.D) : 1.f;
  cp_async_wait<0>();
  __syncthreads();
  const int base = warp * (DP_TT / 4);
  float hist[TAPS][4];
#pragma unroll
  for (int j = 1; j < TAPS; ++j) load_n<__nv_bfloat16, 4>(&x_s[base + TAPS - 1 - j][cl], hist[j]);
#pragma unroll 4
  for (int k = 0; k < DP_TT / 4; ++k) {
    const int t = t0 + base + k;
    if (t >= t1) break;
    load_n<__nv_bfloat16, 4>(&x_s[base + k + TAPS - 1][cl], hist[0]);
    float y[4], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float a = 0.f;
#pragma unroll
      for (int j = TAPS - 1; j >= 0; --j) a = fmaf(w[j][i], hist[j][i], a);
#pragma unroll
      for (int j = TAPS - 1; j > 0; --j) hist[j][i] = hist[j - 1][i];
      y[i] = __bfloat162float(__float2bfloat16(silu_t<__nv_bfloat16>(a)));  // the norm is that of the stored vector
      ss = fmaf(y[i], y[i], ss);
    }
    if (qk) {
      ss = warp_reduce_sum(ss);
      if (lane == 0) p.unit[(long long)(first + t) * 2 * p.Hk + r] = qscale * rsqrtf(ss + UNIT_EPS);
    }
    if (cl < size)
      store_n<__nv_bfloat16, 4>(static_cast<__nv_bfloat16*>(p.qkv) + (long long)(first + t) * C + c0 + cl, y);
  }
}

// The last convolution inputs of a sequence: its channels are dealt out over the `parts` CTAs that work on it.
template <typename T>
__device__ __forceinline__ void store_ring(const DeltaParams& p, int first, int n, int start, int slot, int part, int parts) {
  const int C = 2 * p.Hk * p.D + p.H * p.V;
  const T* proj = static_cast<const T*>(p.proj) + (long long)first * p.stride;
  T* ring = static_cast<T*>(p.ring) + (long long)slot * p.taps * C;
  for (int c = part * blockDim.x + threadIdx.x; c < C; c += parts * blockDim.x)
    for (int t = max(0, n - p.taps); t < n; ++t)
      ring[(long long)((start + t) % p.taps) * C + c] = proj[(long long)t * p.stride + c];
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
  const float* qkv = static_cast<const float*>(p.qkv) + (long long)first * C;
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
  store_ring<T>(p, first, n, start, slot, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
}

// ---------------------------------------------------------------------------------------------------------------
// Chunked form on the tensor cores. Chunk c of sequence b has index (cu_q[b] / 64) + b + c: distinct for all chunks, at
// most T / 64 + B of them.
constexpr int DC = 64;             // tokens per chunk
constexpr int DC_MAT = DC * DC;    // one bf16 term of T or P
// scratch of one (chunk, head): T hi | P T hi | T lo | P T lo (bf16 [64][64] each), then fp32 vectors [64]:
//   e^{G_t} / |k_t|,  e^{G_t} D^{-1/2} / |q_t|,  e^{G_last - G_t} / |k_t|,  e^{G_last} (repeated)
constexpr int DC_VEC_OFF = 4 * DC_MAT * 2;
constexpr int DC_BYTES = DC_VEC_OFF + 4 * DC * 4;

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void mma16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Fragment addresses. A [16 x 16] at (row, col) of a row-major tile:
template <int PITCH>
__device__ __forceinline__ const __nv_bfloat16* frag_a(const __nv_bfloat16* t, int row, int col, int lane) {
  return t + (row + (lane & 15)) * PITCH + col + (lane >> 4) * 8;
}
// B of two neighbouring n-tiles, stored [n][k] (ldsm4)
template <int PITCH>
__device__ __forceinline__ const __nv_bfloat16* frag_bn(const __nv_bfloat16* t, int k, int n, int lane) {
  return t + (n + ((lane >> 4) & 1) * 8 + (lane & 7)) * PITCH + k + ((lane >> 3) & 1) * 8;
}

// One CTA of four warps per (chunk, NH heads that share their q and k): T = (I + A)^-1 diag(beta) and P T of each.
template <int DP, int NH>
struct ChunkPrepSmem {
  static constexpr int PI = DP + 8, AP = DC + 4;
  static constexpr int KQ = 2 * DC * PI * 2, STAGE = NH * 2 * DC_MAT * 2;
  static constexpr int A_OFF = STAGE > KQ ? STAGE : KQ;              // k, q, later P; then A, later T
  static constexpr int G_OFF = A_OFF + NH * DC * AP * 4;
  static constexpr int BYTES = G_OFF + (2 * NH + 2) * DC * 4;
};
template <int DP, int NH>
__global__ void __launch_bounds__(128) delta_chunk_prep_kernel(const DeltaParams p, uint8_t* __restrict__ scratch) {
  using L = ChunkPrepSmem<DP, NH>;
  constexpr int PI = L::PI, AP = L::AP;
  extern __shared__ __align__(16) uint8_t smb[];
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smb);
  __nv_bfloat16* q_s = k_s + DC * PI;
  __nv_bfloat16* p_s = k_s;                                            // P, then P T: NH x (hi | lo)
  float* a_s = reinterpret_cast<float*>(smb + L::A_OFF);               // [NH][64][AP]
  __nv_bfloat16* t_s = reinterpret_cast<__nv_bfloat16*>(smb + L::A_OFF);  // T: NH x (hi | lo)
  float* G_s = reinterpret_cast<float*>(smb + L::G_OFF);               // [NH][64]
  float *b_s = G_s + NH * DC, *nk_s = b_s + NH * DC, *nq_s = nk_s + DC;
  // staged matrices: [64][64] bf16, 16-byte groups swizzled by row
  auto at = [](int m, int t, int c) { return m * DC_MAT + t * DC + (((c >> 3) ^ (t & 7)) << 3) + (c & 7); };
  pdl_trigger();
  pdl_wait();
  const int idx = blockIdx.x, h = blockIdx.y * NH;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int lo = 0, hi = p.B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if ((p.cu_q[mid] >> 6) + mid <= idx) lo = mid; else hi = mid - 1;
  }
  const int b = lo, first = p.cu_q[b], n = p.cu_q[b + 1] - first, t0 = (idx - (first >> 6) - b) * DC;
  if (t0 >= n || p.slots[b] < 0) return;
  const int hk = h / (p.H / p.Hk), C = 2 * p.Hk * p.D + p.H * p.V;
  const __nv_bfloat16* y = static_cast<const __nv_bfloat16*>(p.qkv) + (long long)(first + t0) * C + hk * p.D;
  for (int i = tid; i < DC * (DP / 8); i += 128) {
    const int t = i / (DP / 8), d = i % (DP / 8) * 8;
    const bool on = t0 + t < n && d < p.D;
    const __nv_bfloat16* src = on ? y + (long long)t * C + d : y;
    cp_async16(q_s + t * PI + d, src, on);
    cp_async16(k_s + t * PI + d, src + p.Hk * p.D, on);
  }
  cp_async_commit();
  if (tid < DC) {
    const bool on = t0 + tid < n;
    const long long t = first + t0 + tid;
#pragma unroll
    for (int x = 0; x < NH; ++x) {
      G_s[x * DC + tid] = on ? p.gates[t * 2 * p.H + p.H + h + x] : 0.f;
      b_s[x * DC + tid] = on ? p.gates[t * 2 * p.H + h + x] : 0.f;
    }
    nq_s[tid] = on ? p.unit[t * 2 * p.Hk + hk] : 0.f;
    nk_s[tid] = on ? p.unit[t * 2 * p.Hk + p.Hk + hk] : 0.f;
  }
  __syncthreads();
  if (warp < NH) {  // running sums of the log decays, two tokens per lane
    float* G = G_s + warp * DC;
    const float x0 = G[2 * lane], x1 = G[2 * lane + 1];
    float s = x0 + x1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += v;
    }
    G[2 * lane] = s - x1;
    G[2 * lane + 1] = s;
  }
  cp_async_wait<0>();
  __syncthreads();
  uint8_t* dst = scratch + ((long long)idx * p.H + h) * DC_BYTES;
  if (tid < NH * DC) {
    const int t = tid % DC;
    float* vec = reinterpret_cast<float*>(dst + tid / DC * DC_BYTES + DC_VEC_OFF);
    const float g = G_s[tid], gl = G_s[tid / DC * DC + DC - 1], eg = expf(g);
    vec[t] = eg * nk_s[t];
    vec[DC + t] = eg * nq_s[t];
    vec[2 * DC + t] = expf(gl - g) * nk_s[t];
    vec[3 * DC + t] = expf(gl);
  }
  // Gram matrices of this warp's 16 rows, columns up to the diagonal block
  float kk[8][4] = {}, qk[8][4] = {};
  const int nt_end = 2 * (warp + 1);
#pragma unroll
  for (int k = 0; k < DP / 16; ++k) {
    uint32_t ak[4], aq[4];
    ldsm4(ak, frag_a<PI>(k_s, warp * 16, k * 16, lane));
    ldsm4(aq, frag_a<PI>(q_s, warp * 16, k * 16, lane));
#pragma unroll
    for (int nt = 0; nt < 8; nt += 2) {
      if (nt < nt_end) {
        uint32_t bb[4];
        ldsm4(bb, frag_bn<PI>(k_s, k * 16, nt * 8, lane));
        mma16(kk[nt], ak, bb[0], bb[1]);
        mma16(kk[nt + 1], ak, bb[2], bb[3]);
        mma16(qk[nt], aq, bb[0], bb[1]);
        mma16(qk[nt + 1], aq, bb[2], bb[3]);
      }
    }
  }
  __syncthreads();  // every warp is done with k_s and q_s
#pragma unroll
  for (int x = 0; x < NH; ++x) {
    const float *G = G_s + x * DC, *beta = b_s + x * DC;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = warp * 16 + (lane >> 2) + 8 * half, s = nt * 8 + (lane & 3) * 2;
        float pv[2] = {0.f, 0.f}, av[2] = {0.f, 0.f};
        if (nt < nt_end) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float dec = s + e <= t ? __expf(G[t] - G[s + e]) * nk_s[s + e] : 0.f;
            pv[e] = dec * nq_s[t] * qk[nt][2 * half + e];
            av[e] = s + e < t ? dec * nk_s[t] * beta[t] * kk[nt][2 * half + e] : 0.f;
          }
        }
        uint32_t ph, pl;
        split2(pv[0], pv[1], ph, pl);
        *reinterpret_cast<uint32_t*>(p_s + at(2 * x, t, s)) = ph;
        *reinterpret_cast<uint32_t*>(p_s + at(2 * x + 1, t, s)) = pl;
        *reinterpret_cast<float2*>(a_s + (x * DC + t) * AP + s) = make_float2(av[0], av[1]);
      }
    }
  }
  __syncthreads();
  // forward substitution by blocks of 16 rows: a thread owns one column of (I + A)^-1, whose finished blocks replace the
  // rows of A that have been read (rolled loops: straight-line code for all 64 rows runs at instruction-fetch speed)
  const int col = tid % DC;
  float* A = a_s + (NH == 1 ? 0 : tid / DC) * DC * AP;
  const bool solver = tid < NH * DC;
#pragma unroll 1
  for (int I = 0; I < DC; I += 16) {
    float r[16];
    if (solver) {
#pragma unroll
      for (int e = 0; e < 16; ++e) r[e] = I + e == col ? 1.f : 0.f;
#pragma unroll 1
      for (int k = 0; k < I; k += 4) {
        const float x0 = A[k * AP + col], x1 = A[(k + 1) * AP + col], x2 = A[(k + 2) * AP + col], x3 = A[(k + 3) * AP + col];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const float4 a = *reinterpret_cast<const float4*>(A + (I + e) * AP + k);
          r[e] = fmaf(-a.x, x0, fmaf(-a.y, x1, fmaf(-a.z, x2, fmaf(-a.w, x3, r[e]))));
        }
      }
#pragma unroll
      for (int e = 1; e < 16; ++e)
#pragma unroll
        for (int f = 0; f < e; f += 4) {
          const float4 a = *reinterpret_cast<const float4*>(A + (I + e) * AP + I + f);  // zero from the diagonal on
          r[e] = fmaf(-a.x, r[f], r[e]);
          if (f + 1 < e) r[e] = fmaf(-a.y, r[f + 1], r[e]);
          if (f + 2 < e) r[e] = fmaf(-a.z, r[f + 2], r[e]);
          if (f + 3 < e) r[e] = fmaf(-a.w, r[f + 3], r[e]);
        }
    }
    __syncthreads();  // the rows I .. I + 15 of A are read
    if (solver)
#pragma unroll
      for (int e = 0; e < 16; ++e) A[(I + e) * AP + col] = r[e];
  }
  float x[DC];
  if (solver) {
#pragma unroll
    for (int i = 0; i < DC; ++i) x[i] = A[i * AP + col];  // this thread's own column
  }
  __syncthreads();  // T takes the place of A
  if (solver) {
    const int m = tid / DC * 2;
    const float beta = b_s[tid];
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      const float v = x[i] * beta;
      const __nv_bfloat16 vh = __float2bfloat16(v);
      t_s[at(m, i, col)] = vh;
      t_s[at(m + 1, i, col)] = __float2bfloat16(v - __bfloat162float(vh));
    }
  }
  __syncthreads();
  // P T of this warp's rows, written over its rows of P
#pragma unroll 1
  for (int xh = 0; xh < NH; ++xh) {
    float acc[8][4] = {};
    for (int kt = 0; kt <= warp; ++kt) {
      const int r = warp * 16 + (lane & 15), g = kt * 2 + (lane >> 4), kr = kt * 16 + (lane & 15);
      uint32_t ah[4], al[4];
      ldsm4(ah, p_s + at(2 * xh, r, g * 8));
      ldsm4(al, p_s + at(2 * xh + 1, r, g * 8));
#pragma unroll
      for (int nt = 0; nt < 8; nt += 2) {
        if (nt <= 2 * kt) {  // T is lower triangular
          uint32_t bh[4], bl[4];
          ldsm4t(bh, t_s + at(2 * xh, kr, nt * 8 + (lane >> 4) * 8));
          ldsm4t(bl, t_s + at(2 * xh + 1, kr, nt * 8 + (lane >> 4) * 8));
          mma16(acc[nt], ah, bh[0], bh[1]);
          mma16(acc[nt + 1], ah, bh[2], bh[3]);
          mma16(acc[nt], al, bh[0], bh[1]);
          mma16(acc[nt + 1], al, bh[2], bh[3]);
          mma16(acc[nt], ah, bl[0], bl[1]);
          mma16(acc[nt + 1], ah, bl[2], bl[3]);
        }
      }
    }
    __syncwarp();
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = warp * 16 + (lane >> 2) + 8 * half, s = nt * 8 + (lane & 3) * 2;
        uint32_t ph, pl;
        split2(acc[nt][2 * half], acc[nt][2 * half + 1], ph, pl);
        *reinterpret_cast<uint32_t*>(p_s + at(2 * xh, t, s)) = ph;
        *reinterpret_cast<uint32_t*>(p_s + at(2 * xh + 1, t, s)) = pl;
      }
  }
  __syncthreads();
  // scratch order: T hi, P T hi, T lo, P T lo
  for (int i = tid; i < NH * 4 * DC * 8; i += 128) {
    const int m = i / (DC * 8), t = i / 8 % DC, c = i % 8, head = m >> 2, term = (m >> 1) & 1;
    const __nv_bfloat16* src = (m & 1 ? p_s : t_s) + at(2 * head + term, t, c * 8);
    *reinterpret_cast<uint4*>(dst + head * DC_BYTES + ((m & 3) * DC_MAT + t * DC + c * 8) * 2) =
        *reinterpret_cast<const uint4*>(src);
  }
}

// One CTA of sixteen warps per (sequence, head, 128 state columns); tcgen05 with accumulators in TMEM:
//     RQ [128 = K rows | Q rows, 2 v] = [K; Q] . [S hi | S lo]   (from shared memory; the halves are added when read)
//     rhs                            = v - e^G k S          (rows of K)
//     UO [128, v]                    = [T; P T] . rhs       (rows 0..63 = U, rows 64..127 = P U)
//     S^T [v, d]                    += U'^T . K             (U' = e^{G_last - G} U / |k|, fp32 state in TMEM)
// The MMAs are issued by one thread; between them all warps read their TMEM lanes, scale, split into hi and lo and write
// the next operand. Warp w owns TMEM lanes 32 (w % 4) .. and the 32 columns 32 (w / 4) .. of each accumulator. K and Q of the next chunk arrive
// (and v) while a chunk is worked on, T and P T of the next chunk once UO is done; outputs leave through shared memory, so
// that global accesses are whole rows.
constexpr int DT_THREADS = 512;
constexpr int DT_KQ = 32768;                     // [K; Q]: two 64-column blocks of 128 rows x 128 bytes
constexpr int DT_TP_OFF = 2 * DT_KQ;             // hi | lo, 16 KB each
constexpr int DT_X_OFF = DT_TP_OFF + 32768;      // rhs, then U': hi | lo, [64 tokens][128 columns] in two column blocks
constexpr int DT_S_OFF = DT_X_OFF + 32768;       // S^T [128 v][128 d]: per column block hi | lo
constexpr int DT_V_OFF = DT_S_OFF + 65536;       // two chunks of v [64 tokens][128], 16-byte groups swizzled; then their outputs
constexpr int DT_BAR_OFF = DT_V_OFF + 2 * 16384;
constexpr int DT_SMEM = DT_BAR_OFF + 64 + 1024;

__global__ void __launch_bounds__(DT_THREADS, 1)
delta_chunk_scan_kernel(const DeltaParams p, const uint8_t* __restrict__ scratch, int* status) {
  extern __shared__ uint8_t smb[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smb) + 1023) & ~uintptr_t(1023));
  uint64_t* bar = reinterpret_cast<uint64_t*>(smem + DT_BAR_OFF);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar + 1);
  pdl_wait();
  const int v0 = blockIdx.x * 128, h = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, quad = warp & 3, col0 = (warp >> 2) * 32;
  const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, slot = p.slots[b];
  if (n <= 0 || slot < 0) return;  // uniform for the CTA, before any barrier or allocation
  const int start = p.seq_lens[b] - n, hk = h / (p.H / p.Hk), C = 2 * p.Hk * p.D + p.H * p.V;
  const __nv_bfloat16* y = static_cast<const __nv_bfloat16*>(p.qkv) + (long long)first * C;
  const uint8_t* scr = scratch + ((long long)((first >> 6) + b) * p.H + h) * DC_BYTES;
  const long long scr_step = (long long)p.H * DC_BYTES;
  const int chunks = (n + DC - 1) / DC;
  const int VC = min(128, p.V - v0);             // columns of this CTA

  if (tid == 0) {
    mbar_init(bar, 1);
    mbar_fence_init();
  }
  if (warp == 0) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  auto load_kq = [&](int c) {
    if (c < chunks) {
      uint8_t* dst = smem + (c & 1) * DT_KQ;
      const int t0 = c * DC, groups = p.D > 64 ? 16 : 8;
      for (int i = tid; i < DC * groups; i += DT_THREADS) {
        const int t = i / groups, d = i % groups * 8;
        const bool on = t0 + t < n && d < p.D;
        const __nv_bfloat16* src = y + (on ? (long long)(t0 + t) * C + hk * p.D + d : 0);
        uint8_t* to = dst + (d >> 6) * 16384 + t * 128 + ((((d & 63) >> 3) ^ (t & 7)) << 4);
        cp_async16(to, src + p.Hk * p.D, on);
        cp_async16(to + DC * 128, src, on);
      }
      for (int i = tid; i < DC * 16; i += DT_THREADS) {
        const int t = i >> 4, g = i & 15;
        const bool on = t0 + t < n && g * 8 < VC;
        cp_async16(smem + DT_V_OFF + (c & 1) * 16384 + t * 256 + ((g ^ (t & 7)) << 4),
                   y + (on ? (long long)(t0 + t) * C + 2 * p.Hk * p.D + h * p.V + v0 + g * 8 : 0), on);
      }
    }
    cp_async_commit();
  };
  auto load_tp = [&](int c) {
    if (c < chunks)
      for (int i = tid; i < 256 * 8; i += DT_THREADS) {  // 128 rows of hi, 128 rows of lo
        const int r = i >> 3, g = i & 7;
        cp_async16(smem + DT_TP_OFF + r * 128 + ((g ^ (r & 7)) << 4), scr + c * scr_step + r * 128 + g * 16, true);
      }
    cp_async_commit();
  };
  // 32 fp32 values as two bf16 terms into four 16-byte groups of a 128-byte row, starting at group g0
  auto put32 = [&](uint8_t* hi_row, uint8_t* lo_row, int row, int g0, const float (&f)[32]) {
#pragma unroll
    for (int g = 0; g < 4; ++g) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) split2(f[8 * g + 2 * k], f[8 * g + 2 * k + 1], hi[k], lo[k]);
      const int off = ((g0 + g) ^ (row & 7)) << 4;
      *reinterpret_cast<uint4*>(hi_row + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(lo_row + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
  };
  load_kq(0);
  load_tp(0);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot, my = tmem + ((uint32_t)(quad * 32) << 16);
  const uint32_t RQ = 0, UO = 256, ST = 384;
  pdl_trigger();  // TMEM is held

  // the state: this thread's row v and column half, in steps of 32
  const int row_v = quad * 32 + lane;
  float* st = p.state + (((long long)slot * p.H + h) * p.V + v0 + row_v) * p.D;
  uint8_t* s_hi = smem + DT_S_OFF + (col0 >> 6) * 32768 + row_v * 128;
  const int nd = p.D > 64 ? 128 : 64;            // columns past D are zero
  const bool d_on = col0 < nd;
  const int g0 = (col0 & 32) >> 3;  // first 16-byte group within a 128-byte row
  float egl = __ldg(reinterpret_cast<const float*>(scr + DC_VEC_OFF) + 3 * DC);
  if (d_on) {
    {
      float f[32];
      uint32_t w[32];
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        const int d = col0 + e;
        f[e] = start > 0 && row_v < VC && d < p.D ? st[d] : 0.f;
        w[e] = __float_as_uint(f[e] * egl);
      }
      put32(s_hi, s_hi + 16384, row_v, g0, f);
      tmem_st_32x32(my + ST + col0, w);
    }
    tmem_st_wait();
  }
  cp_async_wait<0>();
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();

  const uint32_t base = smem_u32(smem);
  const int k_steps = (p.D + 15) / 16;
  const uint32_t id_rq = umma_idesc(1, 1, 0, 0, 128, 256);           // A, B K-major
  const uint32_t id_uo = umma_idesc(1, 1, 0, 1, 128, 128);           // B MN-major
  const uint32_t id_s = umma_idesc(1, 1, 1, 1, 128, (uint32_t)nd);   // both MN-major
  uint32_t phase = 0;
  bool ok = true;
  // every thread waits for the MMAs issued last; one failed wait ends the loop for the whole CTA
  auto mma_done = [&](int detail) {
    bool good = false;  // a few products take microseconds: bounded by attempts, without reading the clock
    for (int i = 0; i < (1 << 22) && !good; ++i) good = mbar_try_wait(bar, phase);
    if (!good) report_error(status, ERR_WAIT_TMEM_FULL, detail);
    phase ^= 1;
    tc_fence_after();
    return good;
  };

  // this thread's token (TMEM rows 0..63: K and U, 64..127: Q and O) and its factors, loaded a chunk ahead. Rows of K:
  // e^G / |k| and e^{G_last - G} / |k|; rows of Q: e^G / |q|. next_g: e^{G_last} of the chunk after.
  const int t = (quad & 1) * 32 + lane;
  float next_a = 0.f, next_b = 0.f, next_g = 1.f;
  auto load_vec = [&](int c) {
    if (c < chunks) {
      const float* vec = reinterpret_cast<const float*>(scr + c * scr_step + DC_VEC_OFF);
      next_a = __ldg(vec + (quad < 2 ? 0 : DC) + t);
      next_b = __ldg(vec + 2 * DC + t);
    }
    next_g = c + 1 < chunks ? __ldg(reinterpret_cast<const float*>(scr + (c + 1) * scr_step + DC_VEC_OFF) + 3 * DC) : 1.f;
  };
  load_vec(0);
  auto read_rq = [&](float (&f)[32]) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      uint32_t a[16], l[16];
      tmem_ld_32x16(my + RQ + col0 + 16 * j, a);
      tmem_ld_32x16(my + RQ + 128 + col0 + 16 * j, l);
      tmem_ld_wait();
#pragma unroll
      for (int e = 0; e < 16; ++e) f[16 * j + e] = __uint_as_float(a[e]) + __uint_as_float(l[e]);
    }
  };

  for (int c = 0; c < chunks; ++c) {
    const int t0 = c * DC;
    const uint32_t kq = base + (c & 1) * DT_KQ;
    if (tid == 0) {
      tc_fence_after();
      for (int k = 0; k < k_steps; ++k)
        tc_mma_f16(tmem + RQ, umma_smem_desc(kq + (k >> 2) * 16384 + (k & 3) * 32, 16, 1024),
                   umma_smem_desc(base + DT_S_OFF + (k >> 2) * 32768 + (k & 3) * 32, 16, 1024), id_rq, k != 0);
      tc_commit(bar);
    }
    load_kq(c + 1);
    const float scale_a = next_a, scale_b = next_b, egl_next = next_g;
    load_vec(c + 1);
    ok = mma_done(4 * c) && ok;
    // right-hand side
    uint8_t* vrow = smem + DT_V_OFF + (c & 1) * 16384 + t * 256;
    uint8_t* x_hi = smem + DT_X_OFF + (col0 >> 6) * 8192 + t * 128;
    if (quad < 2) {
      {
        float f[32];
        read_rq(f);
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          const uint4 v4 = *reinterpret_cast<const uint4*>(vrow + (((col0 >> 3) + g) ^ (t & 7)) * 16);
          const uint32_t vw[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int e = 8 * g + 2 * k;
            f[e] = fmaf(-scale_a, f[e], __uint_as_float(vw[k] << 16));
            f[e + 1] = fmaf(-scale_a, f[e + 1], __uint_as_float(vw[k] & 0xffff0000u));
          }
        }
        put32(x_hi, x_hi + 16384, t, g0, f);
      }
    }
    cp_async_wait<1>();  // T and P T of this chunk (the newest group is K and Q of the next one)
    fence_proxy_async_smem();
    tc_fence_before();
    if (!__syncthreads_and(ok)) break;
    if (tid == 0) {
      tc_fence_after();
#pragma unroll 1
      for (int term = 0; term < 3; ++term) {  // hi hi, lo hi, hi lo
        const uint32_t a0 = base + DT_TP_OFF + (term == 1 ? 16384 : 0), b0 = base + DT_X_OFF + (term == 2 ? 16384 : 0);
        for (int k = 0; k < DC / 16; ++k)
          tc_mma_f16(tmem + UO, umma_smem_desc(a0 + k * 32, 16, 1024), umma_smem_desc(b0 + k * 2048, 8192, 1024), id_uo,
                     term != 0 || k != 0);
      }
      tc_commit(bar);
    }
    ok = mma_done(4 * c + 1) && ok;
    {
      uint32_t r[32];
      tmem_ld_32x32(my + UO + col0, r);
      tmem_ld_wait();
      float f[32];
      if (quad < 2) {
#pragma unroll
        for (int e = 0; e < 32; ++e) f[e] = scale_b * __uint_as_float(r[e]);
        put32(x_hi, x_hi + 16384, t, g0, f);
      } else {
        read_rq(f);
#pragma unroll
        for (int e = 0; e < 32; ++e) f[e] = fmaf(scale_a, f[e], __uint_as_float(r[e]));
#pragma unroll
        for (int g = 0; g < 4; ++g)
          *reinterpret_cast<uint4*>(vrow + (((col0 >> 3) + g) ^ (t & 7)) * 16) =
              make_uint4(pack_bf16x2(f[8 * g], f[8 * g + 1]), pack_bf16x2(f[8 * g + 2], f[8 * g + 3]),
                         pack_bf16x2(f[8 * g + 4], f[8 * g + 5]), pack_bf16x2(f[8 * g + 6], f[8 * g + 7]));
      }
    }
    fence_proxy_async_smem();
    tc_fence_before();
    if (!__syncthreads_and(ok)) break;
    if (tid == 0) {
      tc_fence_after();
#pragma unroll 1
      for (int term = 0; term < 2; ++term)
        for (int k = 0; k < DC / 16; ++k)
          tc_mma_f16(tmem + ST, umma_smem_desc(base + DT_X_OFF + term * 16384 + k * 2048, 8192, 1024),
                     umma_smem_desc(kq + k * 2048, 16384, 1024), id_s, 1);
      tc_commit(bar);
    }
    load_tp(c + 1);
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (long long)(first + t0) * p.out_stride + (long long)h * p.V + v0;
    for (int i = tid; i < DC * 16; i += DT_THREADS) {
      const int tt = i >> 4, g = i & 15;
      if (t0 + tt < n && g * 8 < VC)
        *reinterpret_cast<uint4*>(out + (long long)tt * p.out_stride + g * 8) =
            *reinterpret_cast<const uint4*>(smem + DT_V_OFF + (c & 1) * 16384 + tt * 256 + ((g ^ (tt & 7)) << 4));
    }
    ok = mma_done(4 * c + 2) && ok;
    const bool last = c + 1 == chunks;
    if (d_on && ok) {
      {
        uint32_t r[32];
        tmem_ld_32x32(my + ST + col0, r);
        tmem_ld_wait();
        float f[32];
#pragma unroll
        for (int e = 0; e < 32; ++e) f[e] = __uint_as_float(r[e]);
        if (last) {
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            const int d = col0 + e;
            if (row_v < VC && d < p.D) st[d] = f[e];
          }
        } else {
          put32(s_hi, s_hi + 16384, row_v, g0, f);
#pragma unroll
          for (int e = 0; e < 32; ++e) r[e] = __float_as_uint(f[e] * egl_next);
          tmem_st_32x32(my + ST + col0, r);
        }
      }
      tmem_st_wait();
    }
    cp_async_wait<1>();  // K and Q of the next chunk (the newest group is its T and P T)
    fence_proxy_async_smem();
    tc_fence_before();
    if (!__syncthreads_and(ok)) break;
  }
  cp_async_wait<0>();
  if (ok) store_ring<__nv_bfloat16>(p, first, n, start, slot, blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
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
  const float inv = rsqrtf(warp_reduce_sum(ss) * (1.f / (float)p.V) + p.eps);
  const T* gate = proj + C + (long long)h * p.V;
  const T* w = static_cast<const T*>(p.norm_w);
  for (int c = tid; c < p.V; c += DD_THREADS) out[c] = dl_t<T>(o_s[c] * inv * dl_f<T>(w[c]) * silu_f(dl_f<T>(gate[c])));
}

template <typename T>
static int run_prep(const DeltaParams& p, int max_q, cudaStream_t stream) {
  const dim3 g((max_q + DP_TT - 1) / DP_TT, (2 * p.Hk + p.H + DP_GATE_ROWS + 3) / 4, p.B), b(128);
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

template <int DP, int NH>
static cudaError_t launch_chunk_prep(const DeltaParams& p, int tokens, uint8_t* scratch, cudaStream_t stream) {
  constexpr int bytes = ChunkPrepSmem<DP, NH>::BYTES;
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(delta_chunk_prep_kernel<DP, NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return vb_launch_pdl(delta_chunk_prep_kernel<DP, NH>, dim3(tokens / DC + p.B, p.H / NH), dim3(128), bytes, stream, 1, p,
                       scratch);
}

static int run_chunks(const DeltaParams& p, int tokens, uint8_t* scratch, int* status, cudaStream_t stream) {
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(delta_chunk_scan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, DT_SMEM));
    attr = true;
  }
  const bool pairs = (p.H / p.Hk) % 2 == 0;
  cudaError_t e = p.D <= 64 ? (pairs ? launch_chunk_prep<64, 2>(p, tokens, scratch, stream)
                                     : launch_chunk_prep<64, 1>(p, tokens, scratch, stream))
                            : (pairs ? launch_chunk_prep<128, 2>(p, tokens, scratch, stream)
                                     : launch_chunk_prep<128, 1>(p, tokens, scratch, stream));
  if (e != cudaSuccess) return (int)e;
  e = vb_launch_pdl(delta_chunk_scan_kernel, dim3((p.V + 127) / 128, p.H, p.B), dim3(DT_THREADS), DT_SMEM, stream, 1, p,
                    (const uint8_t*)scratch, status);
  vb_count_launch(2);
  return (int)e;
}

template <typename T>
static int run_delta(const DeltaParams& p, int tokens, int max_q, uint8_t* chunk_scratch, int* status,
                     cudaStream_t stream) {
  const int nr = p.D <= 32 ? 4 : p.D <= 64 ? 8 : p.D <= 128 ? 16 : 32;
  if (max_q == 1) {
    if (nr == 4) return run_step<T, 4>(p, stream);
    if (nr == 8) return run_step<T, 8>(p, stream);
    if (nr == 16) return run_step<T, 16>(p, stream);
    return run_step<T, 32>(p, stream);
  }
  int rc;
  if (chunk_scratch) {
    const dim3 g((max_q + DP_TT - 1) / DP_TT, 2 * p.Hk + p.H * ((p.V + 127) / 128) + 1, p.B);
    rc = (int)(p.taps <= 4 ? vb_launch_pdl(delta_prep_tile_kernel<4>, g, dim3(128), 0, stream, 1, p)
                           : vb_launch_pdl(delta_prep_tile_kernel<8>, g, dim3(128), 0, stream, 1, p));
    vb_count_launch();
  } else {
    rc = run_prep<T>(p, max_q, stream);
  }
  if (rc) return rc;
  if (chunk_scratch)
    rc = run_chunks(p, tokens, chunk_scratch, status, stream);
  else
    rc = nr == 4    ? run_scan<T, 4>(p, stream)
         : nr == 8  ? run_scan<T, 8>(p, stream)
         : nr == 16 ? run_scan<T, 16>(p, stream)
                    : run_scan<T, 32>(p, stream);
  if (rc) return rc;
  const T* gate = static_cast<const T*>(p.proj) + 2 * p.Hk * p.D + p.H * p.V;
  return launch_gated_norm<T>(static_cast<T*>(p.out), p.out_stride, gate, p.stride, p.norm_w, p.H, p.V, p.eps, tokens, stream);
}

}  // namespace vb

using namespace vb;

// 1 if the chunked form serves these sizes (bf16 only).
extern "C" int vb_delta_chunk_supported(int D, int V) {
  return D >= 8 && D <= 128 && (D & 7) == 0 && V >= 8 && V <= 256 && (V & 7) == 0;
}
// Bytes of chunk_scratch for T tokens of B sequences.
extern "C" long long vb_delta_chunk_bytes(int T, int B, int H) { return (long long)(T / DC + B) * H * DC_BYTES; }

// Limits: D, V <= 256, taps <= 8. max_q == 1 (every sequence brings exactly one token) takes the fused step and needs no
// scratch. Otherwise gates is fp32 scratch [T, 2 H] and qkv scratch [T, 2 Hk D + H V]: fp32 for the token-by-token scan
// (chunk_scratch and unit null), bf16 for the chunked form, with unit fp32 [T, 2 Hk] and chunk_scratch (16-byte aligned).
extern "C" int vb_delta_rule(const void* proj, long long stride, const void* conv_w, const float* a_log,
                             const float* dt_bias, const void* norm_w, void* ring, float* state, const int* cu_q,
                             const int* seq_lens, const int* slots, void* qkv, float* unit, float* gates, void* chunk_scratch,
                             void* out, long long out_stride, int T, int B, int max_q, int H, int Hk, int D, int V, int taps,
                             float eps, int f32, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_q <= 0) return 0;
  if (Hk <= 0 || H % Hk != 0 || D <= 0 || D > 256 || V <= 0 || V > 256 || taps < 1 || taps > 8 || B > 65535) return -3;
  if (max_q > 1 && (qkv == nullptr || gates == nullptr)) return -3;
  if (max_q > 1 && chunk_scratch != nullptr &&
      (f32 || unit == nullptr || !vb_delta_chunk_supported(D, V) || (out_stride & 7) || (stride & 7) || (reinterpret_cast<uintptr_t>(qkv) & 15)))
    return -3;
  DeltaParams p{proj, stride, conv_w, a_log, dt_bias, norm_w, ring, state, cu_q, seq_lens, slots, qkv, unit, gates, out,
                out_stride, B, H, Hk, D, V, taps, eps};
  uint8_t* scr = reinterpret_cast<uint8_t*>(chunk_scratch);
  const int rc = f32 ? run_delta<float>(p, T, max_q, nullptr, status, stream) : run_delta<__nv_bfloat16>(p, T, max_q, scr, status, stream);
  return rc ? rc : (int)cudaGetLastError();
}
