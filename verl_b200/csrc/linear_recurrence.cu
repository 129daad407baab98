// Gated linear recurrent unit (ops/lru.py) over ragged batches with per-sequence state.
//
//   u = causal convolution of the recurrent branch (+ bias)              lru_conv
//   r, i = sigmoid(block-wise projections of u + bias)
//   a = exp(-power softplus(lam) r),  v = i u sqrt(1 - a a)
//   S = a S + v  token by token,  out = S gelu(gelu branch)
//
// lru_tc does all behind the convolution in one kernel (bf16). A CTA owns 128 channels of a block and walks a sequence, 64 tokens
// at a time: Z^T[channels x tokens] = G[128 channels x n] . u^T on tcgen05 for both gates (weights stay in shared memory, tiles of
// u and of the gelu branch arrive by TMA), then thread = channel: the terms of 16 tokens in registers, one dependent multiply-add
// per token, the carry handed through shared memory to the four warps that hold the next 16 tokens. Neither gates nor decays
// reach memory. Steps of single tokens use the same kernel with sequences in place of tokens and the state in memory in place of the carry.
// lru_gates and lru_scan are the same on CUDA cores (fp32, and sizes the other does not take).
// Every wait is bounded; on expiry the status word is set and the CTA leaves through its teardown.
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

// u[t, c] = bias[c] + sum over j of x[t - taps + 1 + j, c] w[c, j]. Thread: V channels, LC_TOKENS tokens in a row, whose earlier
// inputs stay in registers (TAPS > 0). The row of a single token goes to its sequence's ring here; longer portions write theirs
// behind the scan (other tokens still read the ring).
constexpr int LC_TOKENS = 16, LC_AHEAD = 8;
template <typename T, int V, int TAPS>
__global__ void lru_conv_kernel(const T* __restrict__ proj, const T* __restrict__ w, const T* __restrict__ bias,
                                T* __restrict__ ring, T* __restrict__ u, const int run, const LruParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= p.W) return;
  const T* x = proj + p.W;
  const int t0 = blockIdx.x * run, t1 = min(t0 + run, p.T), taps = TAPS > 0 ? TAPS : p.taps;
  int b = seq_of(p.cu_q, p.B, t0);
  int first = 0, n_new = 0, start = 0, slot = 0;
  // input of token t's row `at` (before the portion: from the ring; before the sequence, or without a slot: zero)
  auto load = [&](int at, float (&f)[V]) {
    const T* src = nullptr;
    if (at >= first) {
      src = x + at * p.stride + c;
    } else if (start + at - first >= 0 && slot >= 0) {
      src = ring + ((long long)slot * taps + (start + at - first) % taps) * p.W + c;
    }
    if (src == nullptr) {
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] = 0.f;
    } else {
      if constexpr (V == 8) ld8(src, f); else f[0] = to_f<T>(src[0]);
    }
  };
  float bias_r[V];
#pragma unroll
  for (int e = 0; e < V; ++e) bias_r[e] = to_f<T>(bias[c + e]);
  float wr[TAPS > 0 ? TAPS : 1][V], hist[TAPS > 1 ? TAPS - 1 : 1][V];
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int e = 0; e < V; ++e) wr[j][e] = to_f<T>(w[(long long)(c + e) * TAPS + j]);
  }
  // u of token t from its input f and the inputs before it
  auto shift = [&](int t, const float (&f)[V]) {
    float acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      acc[e] = bias_r[e];
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) acc[e] = fmaf(hist[j][e], wr[j][e], acc[e]);
      acc[e] = fmaf(f[e], wr[TAPS > 0 ? TAPS - 1 : 0][e], acc[e]);
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j) hist[j][e] = hist[j + 1][e];
      if (TAPS > 1) hist[TAPS > 1 ? TAPS - 2 : 0][e] = f[e];
    }
    if constexpr (V == 8) st8(u + (long long)t * p.W + c, acc); else u[(long long)t * p.W + c] = from_f<T>(acc[0]);
  };
  bool fresh = true;
  for (int t = t0; t < t1; ++t) {
    if (fresh || p.cu_q[b + 1] <= t) {
      while (p.cu_q[b + 1] <= t) ++b;
      first = p.cu_q[b];
      n_new = p.cu_q[b + 1] - first;
      start = p.seq_lens[b] - n_new;
      slot = p.slots[b];
      if constexpr (TAPS > 1) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) load(t - (TAPS - 1) + j, hist[j]);
      }
      fresh = false;
    }
    if constexpr (TAPS > 0 && V == 8 && sizeof(T) == 2) {
      if (t + LC_AHEAD <= t1 && t + LC_AHEAD <= first + n_new && n_new > 1) {  // several inputs on their way at once
        uint4 raw[LC_AHEAD];
#pragma unroll
        for (int i = 0; i < LC_AHEAD; ++i) raw[i] = __ldg(reinterpret_cast<const uint4*>(x + (t + i) * p.stride + c));
#pragma unroll
        for (int i = 0; i < LC_AHEAD; ++i) {
          float f[V];
          ld8(reinterpret_cast<const T*>(&raw[i]), f);
          shift(t + i, f);
        }
        t += LC_AHEAD - 1;
        continue;
      }
    }
    float f[V];
    if constexpr (TAPS > 0) {
      load(t, f);
      shift(t, f);
    } else {
      float acc[V];
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = bias_r[e];
      for (int j = 0; j < taps; ++j) {
        load(t - taps + 1 + j, f);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(f[e], to_f<T>(w[(long long)(c + e) * taps + j]), acc[e]);
      }
      if constexpr (V == 8) st8(u + (long long)t * p.W + c, acc); else u[(long long)t * p.W + c] = from_f<T>(acc[0]);
    }
    if (n_new == 1 && slot >= 0) {
      T* dst = ring + ((long long)slot * taps + start % taps) * p.W + c;
      if constexpr (V == 8) {
        load(t, f);
        st8(dst, f);
      } else {
        dst[0] = x[t * p.stride + c];
      }
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

// Decays and inputs [2, T, W] on the CUDA cores. One block per token and 128 channels. gates null: ab holds the products.
template <typename T>
__global__ void lru_gates_kernel(const T* __restrict__ u, const T* __restrict__ gates, float* __restrict__ ab, const LruParams p) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.W) return;
  const T* ut = u + (long long)blockIdx.x * p.W;
  float *pa = ab + (long long)blockIdx.x * p.W + c, *pv = pa + (long long)p.T * p.W;
  float zr = p.gates_b[c], zi = p.gates_b[p.W + c];
  if (gates) {
    const T *gr = gates + (long long)c * p.n, *gi = gr + (long long)p.W * p.n, *ub = ut + c / p.n * p.n;
    for (int k = 0; k < p.n; ++k) {
      const float f = to_f<T>(ub[k]);
      zr = fmaf(f, to_f<T>(gr[k]), zr);
      zi = fmaf(f, to_f<T>(gi[k]), zi);
    }
  } else {
    zr += *pa;
    zi += *pv;
  }
  lru_terms(zr, zi, to_f<T>(ut[c]), -p.power * softplus_f(p.lam[c]), *pa, *pv);
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

// ------------------------------------------------------------------------------------------------ gates and recurrence, tcgen05
constexpr int LT_COLS = 16;  // tokens of a group of four warps
constexpr int LT_MAX_STAGES = 3, LT_TOKENS = 64, LT_STEP_TOKENS = 32;
constexpr float LT_LOG2E = 1.4426950408889634f;

template <int NT>
struct LtCfg {
  static constexpr int GROUPS = NT / LT_COLS, EPI = 4 * GROUPS, THREADS = (EPI + 2) * 32;
  static constexpr int KB_W = 128 * 128, KB_U = NT * 128;  // bytes of 64 columns of a gate's weights, of a tile of u
  static constexpr int TMEM = 4 * NT;                      // two stages of both gates' logits
  static constexpr int TAIL = 512 + GROUPS * 128 * 4;      // barriers, carries
  // a stage: the block's columns of u, 128 of the gelu branch
  static __host__ __device__ int stage(int kb) { return (kb + 2) * KB_U; }
  static __host__ __device__ int bytes(int kb, int stages) { return 2 * kb * KB_W + stages * stage(kb) + TAIL + 1024; }
};

struct LruTcParams {
  LruParams l;
  const __nv_bfloat16* proj;
  __nv_bfloat16 *ring, *out;
  int kb, tiles, stages, seq0;  // 64-column parts of a block, 128-channel tiles of a block, first sequence
  int steps;                    // STEP: rows (one token each)
  int* status;
};

__device__ __forceinline__ float sqrt_approx(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// The terms of the recurrence from the gates' logits and the input, and the gelu branch; nr, ni = the logits times -log2(e),
// cl = -power * softplus(lam) * log2(e). The three sigmoids share one reciprocal: their denominators are bounded so that the
// product stays finite (below e^-28 a sigmoid is nothing beside what it is added to or multiplied with here).
__device__ __forceinline__ void lru_terms_fast(float nr, float ni, float u, float g, float cl, float& a, float& v, float& y) {
  constexpr float K1 = -2.f * LT_LOG2E * 0.7978845608028654f, K3 = K1 * 0.044715f;
  const float A = 1.f + ex2_approx(fminf(nr, 40.f)), B = 1.f + ex2_approx(fminf(ni, 40.f)),
              C = 1.f + ex2_approx(fminf(g * fmaf(K3, g * g, K1), 40.f));
  const float ab = A * B, q = rcp_approx(ab * C), qc = q * C;
  y = g * (q * ab);
  const float la = cl * (qc * B);  // log2 of the decay
  a = ex2_approx(la);
  // 1 - a^2 = -expm1(x), x = 2 ln(2) la: by its series near zero, where the difference would cancel
  const float x = 1.3862943611198906f * la;
  float e = fmaf(x, 1.f / 5040.f, 1.f / 720.f);
  e = fmaf(x, e, 1.f / 120.f);
  e = fmaf(x, e, 1.f / 24.f);
  e = fmaf(x, e, 1.f / 6.f);
  e = fmaf(x, e, 0.5f);
  e = fmaf(x, e, 1.f);
  const float s = x > -0.3f ? -x * e : fmaf(-a, a, 1.f);
  v = sqrt_approx(s) * (qc * A) * u;
}

template <int NT, bool STEP>
__global__ void __launch_bounds__(LtCfg<NT>::THREADS, 1)
lru_tc_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmU,
              const __grid_constant__ CUtensorMap tmY, const LruTcParams p) {
  using Cfg = LtCfg<NT>;
  constexpr int GROUPS = Cfg::GROUPS, EPI = Cfg::EPI;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int kb = p.kb, stages = p.stages, u_off = 2 * kb * Cfg::KB_W, stage_bytes = Cfg::stage(kb);
  uint64_t* w_full = reinterpret_cast<uint64_t*>(smem + u_off + stages * stage_bytes);
  uint64_t *u_full = w_full + 1, *u_empty = u_full + LT_MAX_STAGES, *t_full = u_empty + LT_MAX_STAGES, *t_empty = t_full + 2,
           *carry = t_empty + 2;  // carry[group * 4 + warp of the group]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(carry + EPI);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* carry_s = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(w_full) + 512);  // [group][channel]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int blk = blockIdx.x / p.tiles, m0 = (blockIdx.x - blk * p.tiles) * 128;  // first channel of the tile in its block
  const int W = p.l.W, n = p.l.n;

  pdl_wait();
  int b = 0, first, nq;
  if (STEP) {
    first = blockIdx.y * NT;
    nq = min(p.steps - first, NT);
  } else {
    b = p.seq0 + blockIdx.y;
    first = p.l.cu_q[b];
    nq = p.l.cu_q[b + 1] - first;
  }
  if (nq <= 0) return;  // uniform for the CTA, before any barrier or allocation
  const int chunks = (nq + NT - 1) / NT;

  if (tid == 0) {
    mbar_init(w_full, 1);
    for (int s = 0; s < LT_MAX_STAGES; ++s) {
      mbar_init(&u_full[s], 1);
      mbar_init(&u_empty[s], EPI);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&t_full[i], 1);
      mbar_init(&t_empty[i], EPI);
    }
    for (int i = 0; i < EPI; ++i) mbar_init(&carry[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == EPI + 1) {
    tmem_alloc(tmem_slot, Cfg::TMEM);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;  // stage s: decay logits at s * 2 NT, input logits NT behind them
  pdl_trigger();

  if (warp == EPI) {
    // ------------------------------- TMA producer -------------------------------
    if (elect_one()) {
      const int blocks = W / n;
      mbar_arrive_expect_tx(w_full, 2 * kb * Cfg::KB_W);
      for (int g = 0; g < 2; ++g)
        for (int k = 0; k < kb; ++k)
          tma_load_3d(smem + (g * kb + k) * Cfg::KB_W, &tmW, w_full, k * 64, m0, g * blocks + blk);
      int c = 0;
      for (; c < chunks; ++c) {
        const int s = c % stages;
        if (*abort_flag || !mbar_wait(&u_empty[s], ((c / stages) & 1) ^ 1)) {
          report_error(p.status, ERR_WAIT_EMPTY, c);
          *abort_flag = 1;
          break;
        }
        uint8_t* dst = smem + u_off + s * stage_bytes;
        mbar_arrive_expect_tx(&u_full[s], stage_bytes);
        for (int k = 0; k < kb; ++k) tma_load_3d(dst + k * Cfg::KB_U, &tmU, &u_full[s], k * 64, blk, first + c * NT);
        for (int k = 0; k < 2; ++k)
          tma_load_2d(dst + (kb + k) * Cfg::KB_U, &tmY, &u_full[s], blk * n + m0 + k * 64, first + c * NT);
      }
      // no copy is in flight when the CTA ends, whatever ended it
      mbar_wait(w_full, 0);
      for (int i = max(c - stages, 0); i < c; ++i) mbar_wait(&u_full[i % stages], (i / stages) & 1);
    }
  } else if (warp == EPI + 1) {
    // -------------------------------- MMA issuer --------------------------------
    if (elect_one()) {
      constexpr uint32_t idesc = umma_idesc(1, 1, 0, 0, 128, NT);  // A = weights, B = u, both K-major
      const uint32_t w_addr = smem_u32(smem), u_addr = w_addr + u_off;
      const int k_steps = (n + 15) / 16;
      bool ok = mbar_wait(w_full, 0);
      for (int c = 0; c < chunks; ++c) {
        const int s = c % stages;
        if (!ok || *abort_flag || !mbar_wait(&u_full[s], (c / stages) & 1) ||
            !mbar_wait(&t_empty[c & 1], ((c >> 1) & 1) ^ 1)) {
          report_error(p.status, ERR_WAIT_FULL, c);
          *abort_flag = 1;
          break;
        }
        tc_fence_after();
        for (int g = 0; g < 2; ++g)
          for (int k = 0; k < k_steps; ++k)
            tc_mma_f16(tmem + (c & 1) * 2 * NT + g * NT,
                       umma_smem_desc(w_addr + (g * kb + (k >> 2)) * Cfg::KB_W + (k & 3) * 32, 16, 1024),
                       umma_smem_desc(u_addr + s * stage_bytes + (k >> 2) * Cfg::KB_U + (k & 3) * 32, 16, 1024), idesc, k != 0);
        tc_commit(&t_full[c & 1]);
      }
    }
  } else {
    // ----------------------- gates and recurrence (thread = channel) -----------------------
    const int group = warp >> 2, quad = warp & 3, row = quad * 32 + lane;  // row: channel of the tile
    const bool on = m0 + row < n;
    const int kc = on ? m0 + row : 0, ch = blk * n + kc;  // channel of the block, of the layer
    const float br = -LT_LOG2E * p.l.gates_b[ch], bi = -LT_LOG2E * p.l.gates_b[W + ch],
                cl = -p.l.power * softplus_f(p.l.lam[ch]) * LT_LOG2E;
    const uint32_t t_addr = tmem + (((uint32_t)(quad * 32)) << 16) + group * LT_COLS;
    // tiles are swizzled: element (row r, column k of a 64-column part) lies at (r / 8) * 1024 + (r % 8) * 128, in 16-byte piece
    // (k / 8) ^ (r % 8); this group's rows start at a multiple of 8
    const uint8_t *u_src = smem + u_off + (kc >> 6) * Cfg::KB_U + group * (LT_COLS / 8) * 1024 + (kc & 7) * 2,
                  *y_src = smem + u_off + (kb + (row >> 6)) * Cfg::KB_U + group * (LT_COLS / 8) * 1024 + (row & 7) * 2;
    const int cu = (kc & 63) >> 3, cy = (row & 63) >> 3;
    int slot = 0, len = 0;
    float S = 0.f, S0[STEP ? LT_COLS : 1];
    if constexpr (STEP) {  // state of the sequences, on its way while the gates are computed
#pragma unroll
      for (int j = 0; j < LT_COLS; ++j) {
        const int t = first + group * LT_COLS + j;
        S0[j] = 0.f;
        if (t < first + nq && on) {
          const int sl = p.l.slots[t];
          if (sl >= 0 && p.l.seq_lens[t] > 1) S0[j] = p.l.state[(long long)sl * W + ch];
        }
      }
    } else {
      slot = p.l.slots[b];
      len = p.l.seq_lens[b];
      if (group == 0 && slot >= 0 && len > nq) S = p.l.state[(long long)slot * W + ch];
    }
    bool ok = true;
    for (int c = 0; c < chunks; ++c) {
      const int s = c % stages, tok0 = c * NT + group * LT_COLS, live = max(min(nq - tok0, LT_COLS), 0);
      if (*abort_flag || !mbar_wait(&u_full[s], (c / stages) & 1) || !mbar_wait(&t_full[c & 1], (c >> 1) & 1)) {
        report_error(p.status, ERR_WAIT_TMEM_FULL, c);
        *abort_flag = 1;
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);  // the lanes of a warp share its TMEM accesses: they stop together
      if (!ok) break;
      tc_fence_after();
      float a[LT_COLS], v[LT_COLS], y[LT_COLS];
      {
        uint32_t zr[LT_COLS], zi[LT_COLS];
        tmem_ld_32x16(t_addr + (c & 1) * 2 * NT, zr);
        tmem_ld_32x16(t_addr + (c & 1) * 2 * NT + NT, zi);
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&t_empty[c & 1]);
        const uint8_t *us = u_src + s * stage_bytes, *ys = y_src + s * stage_bytes;
#pragma unroll
        for (int j = 0; j < LT_COLS; ++j) {
          const int at = (j >> 3) * 1024 + (j & 7) * 128;
          const float u = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(us + at + ((cu ^ (j & 7)) << 4)));
          const float g = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(ys + at + ((cy ^ (j & 7)) << 4)));
          lru_terms_fast(fmaf(__uint_as_float(zr[j]), -LT_LOG2E, br), fmaf(__uint_as_float(zi[j]), -LT_LOG2E, bi), u, g, cl, a[j],
                         v[j], y[j]);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&u_empty[s]);
      if constexpr (STEP) {
#pragma unroll
        for (int j = 0; j < LT_COLS; ++j) {
          if (j < live && on) {
            const int t = first + tok0 + j, sl = p.l.slots[t];
            const float S1 = fmaf(a[j], S0[j], v[j]);
            if (sl >= 0) p.l.state[(long long)sl * W + ch] = S1;
            p.out[(long long)t * W + ch] = __float2bfloat16(sl >= 0 ? S1 * y[j] : 0.f);
          }
        }
        continue;
      }
      if (live < LT_COLS) {  // past the portion the state stays
#pragma unroll
        for (int j = 0; j < LT_COLS; ++j)
          if (j >= live) {
            a[j] = 1.f;
            v[j] = 0.f;
          }
      }
      if (group > 0 || c > 0) {  // from the group that holds the tokens before these
        const int from = group > 0 ? group - 1 : GROUPS - 1;
        if (*abort_flag || !mbar_wait(&carry[from * 4 + quad], (group > 0 ? c : c - 1) & 1)) {
          report_error(p.status, ERR_WAIT_FLAG, c);
          *abort_flag = 1;
          ok = false;
        }
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        S = carry_s[from * 128 + row];
      }
#pragma unroll
      for (int j = 0; j < LT_COLS; ++j) {
        S = fmaf(a[j], S, v[j]);
        a[j] = S;
      }
      carry_s[group * 128 + row] = S;
      __syncwarp();
      if (lane == 0) mbar_arrive(&carry[group * 4 + quad]);
      __nv_bfloat16* dst = p.out + (long long)(first + tok0) * W + ch;
      if (on) {
        if (live == LT_COLS && slot >= 0) {
#pragma unroll
          for (int j = 0; j < LT_COLS; ++j, dst += W) *dst = __float2bfloat16(a[j] * y[j]);
        } else {
#pragma unroll
          for (int j = 0; j < LT_COLS; ++j, dst += W)
            if (j < live) *dst = __float2bfloat16(slot >= 0 ? a[j] * y[j] : 0.f);
        }
      }
    }
    if (!STEP && ok && group == GROUPS - 1 && on && slot >= 0) {  // S: behind the last token
      p.l.state[(long long)slot * W + ch] = S;
      if (nq > 1) write_ring<__nv_bfloat16>(p.proj + W, p.ring, p.l, first, nq, len, slot, ch);
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == EPI + 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::TMEM);
  }
}

}  // namespace vb

using namespace vb;
typedef __nv_bfloat16 bf16;

template <typename T, int V>
static cudaError_t launch_conv(const void* proj, const void* w, const void* bias, void* ring, void* u, const LruParams& p,
                               cudaStream_t stream) {
  const int threads = p.W / V >= 256 ? 128 : 64;
  const int run = p.T >= 8 * p.B ? LC_TOKENS : 1;  // mostly single tokens: nothing to keep from one to the next
  const dim3 g((p.T + run - 1) / run, (p.W / V + threads - 1) / threads);
#define VB_LC(N)                                                                                                              \
  vb_launch_pdl(lru_conv_kernel<T, V, N>, g, dim3(threads), 0, stream, 1, (const T*)proj, (const T*)w, (const T*)bias, (T*)ring, \
                (T*)u, run, p)
  vb_count_launch();
  switch (p.taps) {
    case 1: return VB_LC(1);
    case 2: return VB_LC(2);
    case 3: return VB_LC(3);
    case 4: return VB_LC(4);
    default: return VB_LC(0);
  }
#undef VB_LC
}

template <typename T>
static int rglru_simt(const void* proj, const void* gates, void* ring, const void* u, float* ab, void* out, const LruParams& p,
                      cudaStream_t stream) {
  cudaError_t e = vb_launch_pdl(lru_gates_kernel<T>, dim3(p.T, (p.W + 127) / 128), dim3(128), 0, stream, 1, (const T*)u,
                                (const T*)gates, ab, p);
  vb_count_launch();
  if (e != cudaSuccess) return (int)e;
  VB_DONE(vb_launch_pdl(lru_scan_kernel<T>, dim3((p.W + 63) / 64, p.B), dim3(64), 0, stream, 1, (const T*)proj, (const float*)ab,
                        (T*)ring, (T*)out, p));
}

// Stages of u that fit beside the weights of 64 * kb columns (0: none).
template <int NT>
static int lt_stages(int kb) {
  int s = LT_MAX_STAGES;
  while (s > 0 && LtCfg<NT>::bytes(kb, s) > 227 * 1024) --s;
  return s;
}

extern "C" int vb_rglru_tc_supported(int W, int n) {
  return n > 0 && W % n == 0 && (n & 7) == 0 && lt_stages<LT_TOKENS>((n + 63) / 64) >= 1;
}

template <int NT, bool STEP>
static int launch_tc(const CUtensorMap& tmW, const void* u, LruTcParams p, int rows, cudaStream_t stream) {
  CUtensorMap tmU, tmY;
  const uint64_t n = p.l.n, W = p.l.W;
  int rc = vb_make_tmap_3d(&tmU, u, 2, n, W / n, p.l.T, n * 2, W * 2, 64, 1, NT);
  if (!rc) rc = vb_make_tmap_2d(&tmY, p.proj, 2, W, p.l.T, (uint64_t)p.l.stride * 2, 64, NT);
  if (rc) return rc;
  p.stages = lt_stages<NT>(p.kb);
  if (STEP) p.stages = 1;
  static bool attr_set = false;
  if (!attr_set) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(lru_tc_kernel<NT, STEP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    attr_set = true;
  }
  VB_DONE(vb_launch_pdl(lru_tc_kernel<NT, STEP>, dim3(p.tiles * (p.l.W / p.l.n), rows), dim3(LtCfg<NT>::THREADS),
                        (size_t)LtCfg<NT>::bytes(p.kb, p.stages), stream, 1, tmW, tmU, tmY, p));
}

// u [T, W]: the convolution of the recurrent branch of proj, alone.
extern "C" int vb_rglru_conv(const void* proj, long long stride, const void* conv_w, const void* conv_b, void* ring,
                             const int* cu_q, const int* seq_lens, const int* slots, void* u, int T, int B, int W, int taps, int f32,
                             cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (W <= 0 || taps <= 0) return -3;
  LruParams p{cu_q, seq_lens, slots, T, B, W, W, taps, 0.f, stride, nullptr, nullptr, nullptr};
  const bool vec = (W & 7) == 0 && (stride & 7) == 0;
#define VB_CONV(TT)                                                      \
  (vec ? launch_conv<TT, 8>(proj, conv_w, conv_b, ring, u, p, stream)    \
       : launch_conv<TT, 1>(proj, conv_w, conv_b, ring, u, p, stream))
  const cudaError_t e = f32 ? VB_CONV(float) : VB_CONV(bf16);
#undef VB_CONV
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// Behind vb_rglru_conv. proj [T, stride] (gelu branch | recurrent branch), gates [2, W / n, n, n] (null: ab holds the products of u
// with them), gates_b [2, W], lam [W] fp32, ring [slots, taps, W], state fp32 [slots, W], ab fp32 [2, T, W] scratch (without tc),
// out [T, W]. The leading `singles` sequences have one token each.
extern "C" int vb_rglru(const void* proj, long long stride, const void* gates, const float* gates_b,
                        const float* lam, void* ring, float* state, const int* cu_q, const int* seq_lens, const int* slots, void* u,
                        float* ab, void* out, int T, int B, int singles, int W, int n, int taps, float power, int f32, int tc,
                        int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (W <= 0 || n <= 0 || W % n || taps <= 0 || B > 65535 || (W + 127) / 128 > 65535 || singles < 0 || singles > B ||
      (!tc && ab == nullptr) || (tc && (f32 || gates == nullptr || !vb_rglru_tc_supported(W, n))))
    return -3;
  LruParams p{cu_q, seq_lens, slots, T, B, W, n, taps, power, stride, gates_b, lam, state};
  if (f32) return rglru_simt<float>(proj, gates, ring, u, ab, out, p, stream);
  if (!tc) return rglru_simt<bf16>(proj, gates, ring, u, ab, out, p, stream);
  CUtensorMap tmW;
  const uint64_t n64 = n;
  int rc = vb_make_tmap_3d(&tmW, gates, 2, n64, n64, (uint64_t)(2 * (W / n)), n64 * 2, n64 * n64 * 2, 64, 128, 1);
  if (rc) return rc;
  LruTcParams q{};
  q.l = p;
  q.proj = (const bf16*)proj; q.ring = (bf16*)ring; q.out = (bf16*)out;
  q.kb = (n + 63) / 64; q.tiles = (n + 127) / 128; q.status = status;
  if (singles > 0) {
    q.steps = singles;
    rc = launch_tc<LT_STEP_TOKENS, true>(tmW, u, q, (singles + LT_STEP_TOKENS - 1) / LT_STEP_TOKENS, stream);
    if (rc) return rc;
  }
  if (singles == B) return 0;
  q.seq0 = singles;
  return launch_tc<LT_TOKENS, false>(tmW, u, q, B - singles, stream);
}
