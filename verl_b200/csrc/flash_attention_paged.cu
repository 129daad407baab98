// Prefill attention of layer-list decoders on tcgen05: ragged queries over the paged KV cache, with a sliding window and
// kept first keys or chunks of the sequence, a per-distance bias or a soft cap of the scores, a sink in the denominator and
// an output gate; with softmax weights or sigmoid ones. Head sizes up to 128 (multiples of 8), bf16.
//
// One CTA per (sequence, query head, block of 128 queries), two CTAs per SM: one's softmax overlaps the other's tensor
// work. The CTA walks the 128-key blocks that some row of the block may see: those of the kept first keys, then those of
// the window or chunk. Per block of keys:
//     S[128 q x 128 keys] = Q . K^T                       (tcgen05.mma, accumulator in TMEM)
//     P = exp(S * scale + bias[distance] - reference)     (thread = query row; the soft cap in place of the bias)
//     O[128 q x Dv]      += P . V                         (A operand = P in TMEM, accumulator in TMEM)
// The weights stay close to fp32: P is split into two bf16 terms (P = hi + lo) that are written over the columns of S
// they came from, and both are multiplied with V. A row's reference is a running maximum that only moves when the
// maximum has grown by more than 2^8 (the result does not depend on it), so O is rarely rescaled.
// K / V pages arrive by per-CTA TMA loads; columns past a head's size are filled with zeros by TMA, keys past the sequence
// or outside the mask get weight zero. Masks and the bias table are looked at only by the 32 x 32 blocks they reach.
// The SIG variant weighs a key with the sigmoid of its score, less r1 ln(1 + r2 distance), plus a number of the head, without
// reference, rescaling and denominator. The distance's part of the exponent comes from a table of the 255 distances between 128
// queries and 128 keys, written anew for every block of keys.
// The LATENT variant serves latent attention: keys and values of all heads lie expanded in rows of scratch memory, sequence
// after sequence, and a key is two parts: the head's own and the rotated one that all heads share. Its three 64-column parts
// of Q and K leave room for two CTAs per SM with 64 keys a block. Its contexts may start where the first query's window does:
// only distances count.
// Every wait is bounded; on expiry the status word is set and the CTA leaves through its teardown.
#include "common.cuh"
#include "host_utils.h"

namespace vb {

constexpr int PF_M = 128;                         // queries per CTA
constexpr int PF_THREADS = 192;
constexpr int PF_MAX_BIAS = 3072;                 // distances staged in shared memory
constexpr float PF_SLACK = 8.f;                   // growth of the row maximum (log2) that is let through

template <bool LATENT>
struct PfCfg {
  static constexpr int N = LATENT ? 64 : 128;           // keys per block
  static constexpr int HALVES = LATENT ? 3 : 2;         // 64-column parts of Q and K
  static constexpr int KV_HALF = N * 128;               // bytes of 64 columns of K or V
  static constexpr int K_OFF = HALVES * PF_M * 128;     // Q first, then one K and one V tile
  static constexpr int V_OFF = K_OFF + HALVES * KV_HALF;
  static constexpr int BAR_OFF = V_OFF + 2 * KV_HALF;
  static constexpr int BIAS_OFF = BAR_OFF + 8 * 8 + 32;
};

struct PagedFlashParams {
  const int* cu_q;         // [B + 1]
  const int* seq_lens;     // [B]
  const int* block_table;  // [B, max_blocks]
  const float* bias;       // [Hq, bias_len] or null
  __nv_bfloat16* out;      // [T, out_stride]
  long long out_stride;
  int max_blocks, Hq, Hk, D, Dv, block_size, window, keep_first, chunk, bias_len, max_qblocks;
  float scale, softcap;
  const float* sink;            // [Hq] or null
  const __nv_bfloat16* gate;    // [T, Hq * Dv] (gate_w 1: [T, Hq]) or null
  long long gate_stride;
  int gate_w;
  int* status;
  const float *shift, *r1, *r2;  // [Hq]; SIG: shift, and r1, r2 or null
  // LATENT only: D = the heads' own part of a key; contexts of the sequences in the expanded rows
  int rot;
  const int* ctx_cu;       // [B + 1]
};

// exp2 of the scaled scores: scale and bias are multiplied by log2(e) up front
constexpr float LOG2E = 1.4426950408889634f;

constexpr int PF_TAB = 256;  // distances of a block of keys (SIG), double-buffered in place of the bias table

// Barrier over the 128 threads of the first four warps that also and-reduces a predicate: they leave their loop together.
__device__ __forceinline__ bool pf_bar_and(bool pred) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 q, %1, 0;\n\tbarrier.red.and.pred p, 1, 128, q;\n\tselp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(r)
      : "r"((uint32_t)pred)
      : "memory");
  return r != 0;
}

template <bool LATENT, bool SIG = false>
__global__ void __launch_bounds__(PF_THREADS, 2)
paged_flash_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                   const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmQr,
                   const __grid_constant__ CUtensorMap tmKr, const PagedFlashParams p) {
  using Cfg = PfCfg<LATENT>;
  constexpr int PF_N = Cfg::N, GROUPS = PF_N / 32;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  // barriers: [0] Q, [1] K full, [2] V full, [3] K empty, [4] V empty, [5] S full, [6] P ready, [7] O full
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + Cfg::BAR_OFF);
  uint64_t *q_full = bars, *full = bars + 1, *empty = bars + 3, *s_full = bars + 5, *p_ready = bars + 6, *o_full = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* bias_s = reinterpret_cast<float*>(smem + Cfg::BIAS_OFF);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.z, hq = blockIdx.y;
  pdl_wait();
  const int q_first = p.cu_q[b], n_q = p.cu_q[b + 1] - q_first;
  const int r0 = (p.max_qblocks - 1 - (int)blockIdx.x) * PF_M;  // late blocks (most keys) first
  if (r0 >= n_q) return;  // uniform for the CTA, before any barrier or allocation
  const int hk = hq / (p.Hq / p.Hk);
  const int ctx0 = LATENT ? p.ctx_cu[b] : 0;
  const int seq_len = LATENT ? p.ctx_cu[b + 1] - ctx0 : p.seq_lens[b];
  const int pos0 = seq_len - n_q + r0;                     // position of row 0
  const int pos1 = min(pos0 + PF_M, seq_len) - 1;          // last real row
  const bool windowed = p.window > 0 || (!LATENT && p.chunk > 0);
  const int keep = !LATENT && p.window > 0 ? p.keep_first : 0;
  // first key that a query at position i sees, kept ones apart
  auto first_key = [&](int i) { return LATENT || p.window > 0 ? i - p.window + 1 : i - i % p.chunk; };
  // chunks to visit: [0, keep_chunks) and [win_chunk, last_chunk]
  const int last_chunk = pos1 / PF_N;
  const int keep_chunks = min((keep + PF_N - 1) / PF_N, last_chunk + 1);
  const int win_chunk = max(windowed ? max(first_key(pos0), 0) / PF_N : 0, keep_chunks);
  const int n_chunks = keep_chunks + max(last_chunk + 1 - win_chunk, 0);
  auto chunk_at = [&](int c) { return c < keep_chunks ? c : win_chunk + c - keep_chunks; };

  if (tid == 0) {
    for (int i = 0; i < 8; ++i) mbar_init(&bars[i], i == 6 ? 4 : 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
  }
  if (!LATENT && p.bias != nullptr)
    for (int i = tid; i < p.bias_len; i += PF_THREADS) bias_s[i] = p.bias[(long long)hq * p.bias_len + i] * LOG2E;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;  // S / P: columns 0..127, O: 128..255
  pdl_trigger();  // TMEM is held: a dependent kernel may take what is left
  const int k_halves = p.D > 64 ? 2 : 1, r_halves = LATENT ? (p.rot + 63) / 64 : 0, v_halves = p.Dv > 64 ? 2 : 1;

  if (warp == 4) {
    // ------------------------------- TMA producer -------------------------------
    if (elect_one()) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      mbar_arrive_expect_tx(q_full, (k_halves + r_halves) * 16384);
      for (int x = 0; x < k_halves; ++x) tma_load_3d(smem + x * 16384, &tmQ, q_full, x * 64, hq, q_first + r0);
      for (int x = 0; x < r_halves; ++x)
        tma_load_3d(smem + (k_halves + x) * 16384, &tmQr, q_full, x * 64, hq, q_first + r0);
      const int* bt = LATENT ? nullptr : p.block_table + (long long)b * p.max_blocks;
      const int ppc = LATENT ? 0 : PF_N / p.block_size;
      const int n_pages = LATENT ? 0 : (seq_len + p.block_size - 1) / p.block_size;
      int t = 0;
      for (; t < 2 * n_chunks; ++t) {
        const int s = t & 1;  // 0 = K, 1 = V
        if (*abort_flag || !mbar_wait(&empty[s], ((t >> 1) & 1) ^ 1)) {
          report_error(p.status, ERR_WAIT_EMPTY, t);
          *abort_flag = 1;
          break;
        }
        const int halves = s ? v_halves : k_halves;
        mbar_arrive_expect_tx(&full[s], (halves + (s ? 0 : r_halves)) * Cfg::KV_HALF);
        uint8_t* dst = smem + (s ? Cfg::V_OFF : Cfg::K_OFF);
        const CUtensorMap* tm = s ? &tmV : &tmK;
        if constexpr (LATENT) {  // rows past the context: the next sequence's, or zeros past the last; weight zero
          const int row = ctx0 + chunk_at(t >> 1) * PF_N;
          for (int x = 0; x < halves; ++x) tma_load_3d(dst + x * Cfg::KV_HALF, tm, &full[s], x * 64, hq, row);
          for (int x = 0; x < r_halves && !s; ++x)
            tma_load_2d(dst + (halves + x) * Cfg::KV_HALF, &tmKr, &full[s], x * 64, row);
          continue;
        }
        const int page0 = chunk_at(t >> 1) * ppc;
        for (int pg = 0; pg < ppc; ++pg) {
          // pages past the end re-read the last page: finite data, weight zero
          const int row = (bt[min(page0 + pg, n_pages - 1)] * p.Hk + hk) * p.block_size;
          for (int x = 0; x < halves; ++x)
            tma_load_2d(dst + x * Cfg::KV_HALF + pg * p.block_size * 128, tm, &full[s], x * 64, row);
        }
      }
      // no copy is in flight when the CTA ends, whatever ended it
      mbar_wait(q_full, 0);
      for (int i = max(t - 2, 0); i < t; ++i) mbar_wait(&full[i & 1], (i >> 1) & 1);
    }
  } else if (warp == 5) {
    // -------------------------------- MMA issuer --------------------------------
    if (elect_one()) {
      const uint32_t idesc_qk = umma_idesc(1, 1, 0, 0, PF_M, PF_N);
      const uint32_t idesc_pv = umma_idesc(1, 1, 0, 1, PF_M, (uint32_t)((p.Dv + 15) / 16 * 16));
      const uint32_t q_addr = smem_u32(smem), k_addr = q_addr + Cfg::K_OFF, v_addr = q_addr + Cfg::V_OFF;
      const int k_steps = (p.D + 15) / 16, r_steps = LATENT ? (p.rot + 15) / 16 : 0;
      auto wait = [&](uint64_t* bar, uint32_t parity, int code, int detail) -> bool {
        if (!*abort_flag && mbar_wait(bar, parity)) return true;
        report_error(p.status, code, detail);
        *abort_flag = 1;
        return false;
      };
      bool ok = wait(q_full, 0, ERR_WAIT_FULL, 9000);
      for (int c = 0; ok && c < n_chunks; ++c) {
        ok = wait(&full[0], c & 1, ERR_WAIT_FULL, 2 * c);
        // S takes the place of the previous chunk's P: that chunk's P.V must have completed
        if (ok && c > 0) ok = wait(o_full, (c - 1) & 1, ERR_WAIT_TMEM_EMPTY, 2000 + c);
        if (!ok) break;
        tc_fence_after();
        for (int k = 0; k < k_steps + r_steps; ++k) {
          const int r = k - k_steps;  // step of the rotated part
          const int part = r < 0 ? k >> 2 : k_halves + (r >> 2), in = ((r < 0 ? k : r) & 3) * 32;
          tc_mma_f16(tmem_base, umma_smem_desc(q_addr + part * 16384 + in, 16, 1024),
                     umma_smem_desc(k_addr + part * Cfg::KV_HALF + in, 16, 1024), idesc_qk, k != 0);
        }
        tc_commit(s_full);
        tc_commit(&empty[0]);
        ok = wait(&full[1], c & 1, ERR_WAIT_FULL, 2 * c + 1) && wait(p_ready, c & 1, ERR_WAIT_TMEM_EMPTY, c);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < PF_N / 16; ++k) {
          const uint64_t bv = umma_smem_desc(v_addr + k * 2048, Cfg::KV_HALF, 1024);
          const uint32_t a = tmem_base + (k >> 1) * 32 + (k & 1) * 8;  // per 32 keys: 16 columns of hi, 16 of lo
          tc_mma_f16_ta(tmem_base + 128, a, bv, idesc_pv, c != 0 || k != 0);
          tc_mma_f16_ta(tmem_base + 128, a + 16, bv, idesc_pv, 1);
        }
        tc_commit(o_full);
        tc_commit(&empty[1]);
      }
    }
  } else {
    // ----------------------- softmax (128 threads, thread = query row) -----------------------
    const int r = tid, qpos = pos0 + r, qw = pos0 + warp * 32;  // qw: first row of the warp
    const uint32_t s_addr = tmem_base + (((uint32_t)(warp * 32)) << 16), o_addr = s_addr + 128;
    const float scale2 = p.scale * LOG2E;
    const bool biased = !LATENT && p.bias != nullptr, soft = !LATENT && p.softcap > 0.f;
    // soft cap, in log2 units: cap tanh(z) = cap - 2 cap / (1 + e^(2 z)), z = score / cap
    const float cap2 = p.softcap * LOG2E, cap_k = soft ? 2.f * LOG2E * p.scale / p.softcap : 0.f;
    auto capped = [&](float raw) { return cap2 - __fdividef(2.f * cap2, 1.f + exp2f(raw * cap_k)); };
    // The same for |z| <= 0.7 without the special-function unit, which the exponentials keep busy: an odd polynomial fitted to
    // tanh there (largest error 1e-7). Its coefficients carry cap and scale; they need a range in which z^9 does not underflow.
    const float zs = soft ? p.scale / p.softcap : 0.f, z2 = zs * zs;
    const bool poly_ok = soft && zs > 1e-3f && zs < 1e3f;
    const float k0c = 0.999998495f * cap2 * zs, k1c = -0.33326973f * cap2 * zs * z2, k2c = 0.132574543f * cap2 * zs * z2 * z2,
                k3c = -0.0501952428f * cap2 * zs * z2 * z2 * z2, k4c = 0.0131941733f * cap2 * zs * z2 * z2 * z2 * z2;
    auto capped_small = [&](float raw) {
      const float t = raw * raw;
      return raw * fmaf(t, fmaf(t, fmaf(t, fmaf(t, k4c, k3c), k2c), k1c), k0c);
    };
    const int sat = biased ? p.bias_len - 1 : 0;
    const float bias_far = biased ? bias_s[sat] : 0.f;
    // the sink is a key without a value: its weight starts the denominator
    const bool sunk = p.sink != nullptr;
    float m_ref = sunk ? p.sink[hq] * LOG2E : -INFINITY, l_run = sunk ? 1.f : 0.f;
    const int first = windowed ? first_key(qpos) : 0, first_lo = windowed ? first_key(qw) : 0,
              first_hi = windowed ? first_key(qw + 31) : 0;
    bool ok = true;

    if constexpr (SIG) {
      static_assert(!LATENT, "sigmoid weights over the paged cache only");
      l_run = 1.f;
      const float shift2 = p.shift[hq] * LOG2E, r1 = p.r1 ? p.r1[hq] : 0.f, r2 = p.r1 ? p.r2[hq] : 0.f;
      for (int c = 0; c < n_chunks; ++c) {
        const int c0 = chunk_at(c) * PF_N;
        // what the exponent of e^-(score + shift) takes from the distance d, at entry d - (distance of row 0 to the last key)
        float* tab = bias_s + (c & 1) * PF_TAB;
        for (int i = r; i < PF_TAB; i += 128)
          tab[i] = fmaf(r1, __log2f(fmaf(r2, (float)max(pos0 - c0 - (PF_N - 1) + i, 0), 1.f)), -shift2);
        ok = pf_bar_and(ok);  // the table is complete; a failed wait of the last round ends the loop for all
        if (!ok) break;
        if (*abort_flag || !mbar_wait(s_full, c & 1)) {
          report_error(p.status, ERR_WAIT_TMEM_FULL, c);
          *abort_flag = 1;
          ok = false;
        }
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) continue;  // to the barrier
        tc_fence_after();
        const float* row = tab + r + PF_N - 1;  // entry of key c0 + e: row[-e]
#pragma unroll 1
        for (int j = 0; j < GROUPS; ++j) {
          const int k0 = c0 + 32 * j, dmin = qw - (k0 + 31), dmax = qw + 31 - k0;
          uint32_t v[32];
          if (dmax < 0 || (windowed && k0 + 31 < first_lo && k0 >= keep)) {
#pragma unroll
            for (int e = 0; e < 32; ++e) v[e] = 0;
          } else {
            tmem_ld_32x32(s_addr + j * 32, v);
            tmem_ld_wait();
            uint32_t seen = 0xffffffffu;  // bit e
            if (dmin < 0 || (windowed && k0 < first_hi && k0 + 31 >= keep)) {
              seen = 0;
#pragma unroll
              for (int e = 0; e < 32; ++e)
                seen |= (uint32_t)(qpos >= k0 + e && (!windowed || k0 + e >= first || k0 + e < keep)) << e;
            }
            uint32_t w[32];
#pragma unroll
            for (int e = 0; e < 32; e += 2) {
              // 1 / a and 1 / b from one reciprocal; weights below 2^-60 do not matter
              float x0 = fminf(fmaf(__uint_as_float(v[e]), -scale2, row[-32 * j - e]), 60.f);
              float x1 = fminf(fmaf(__uint_as_float(v[e + 1]), -scale2, row[-32 * j - e - 1]), 60.f);
              x0 = seen >> e & 1 ? x0 : 60.f;
              x1 = seen >> (e + 1) & 1 ? x1 : 60.f;
              const float a = 1.f + exp2f(x0), b = 1.f + exp2f(x1), rc = __fdividef(1.f, a * b);
              const float p0 = seen >> e & 1 ? b * rc : 0.f, p1 = seen >> (e + 1) & 1 ? a * rc : 0.f;
              const uint32_t h = pack_bf16x2(p0, p1);
              w[e >> 1] = h;
              w[16 + (e >> 1)] = pack_bf16x2(p0 - __uint_as_float(h << 16), p1 - __uint_as_float(h & 0xffff0000u));
            }
#pragma unroll
            for (int e = 0; e < 32; ++e) v[e] = w[e];
          }
          tmem_st_32x32(s_addr + j * 32, v);
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_ready);
      }
    } else
    for (int c = 0; c < n_chunks; ++c) {
      if (*abort_flag || !mbar_wait(s_full, c & 1)) {
        report_error(p.status, ERR_WAIT_TMEM_FULL, c);
        *abort_flag = 1;
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);  // the lanes of a warp share its TMEM accesses: they stop together
      if (!ok) break;
      tc_fence_after();
      const int c0 = chunk_at(c) * PF_N;
      // 32-key groups, as this warp sees them: bit j of `none`: nothing visible; of `plain`: all visible, all far
      uint32_t none = 0, plain = 0;
#pragma unroll
      for (int j = 0; j < GROUPS; ++j) {
        const int k0 = c0 + 32 * j, dmin = qw - (k0 + 31), dmax = qw + 31 - k0;
        if (dmax < 0 || (windowed && k0 + 31 < first_lo && k0 >= keep)) none |= 1u << j;
        else if (dmin >= sat && dmin >= 0 && scale2 > 0.f && (!windowed || k0 >= first_hi || k0 + 31 < keep)) plain |= 1u << j;
      }
      // pass 1: row maximum. Blocks with masks or table distances leave their final scores in place of the raw ones.
      float cmax = -INFINITY;
      uint32_t small = 0;  // bit j: every score of the warp's block takes the polynomial
#pragma unroll 1
      for (int j = 0; j < GROUPS; ++j) {
        if (none >> j & 1) continue;
        uint32_t v[32];
        tmem_ld_32x32(s_addr + j * 32, v);
        tmem_ld_wait();
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        if (plain >> j & 1) {
#pragma unroll
          for (int e = 0; e < 32; ++e) mx[e & 3] = fmaxf(mx[e & 3], __uint_as_float(v[e]));
          const float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
          if (soft) {
            float low[4] = {INFINITY, INFINITY, INFINITY, INFINITY};
#pragma unroll
            for (int e = 0; e < 32; ++e) low[e & 3] = fminf(low[e & 3], __uint_as_float(v[e]));
            const float far = fmaxf(fabsf(top), fabsf(fminf(fminf(low[0], low[1]), fminf(low[2], low[3]))));
            small |= (uint32_t)__all_sync(0xffffffffu, poly_ok && far * zs <= 0.7f) << j;
            cmax = fmaxf(cmax, capped(top));
          } else {
            cmax = fmaxf(cmax, fmaf(top, scale2, bias_far));
          }
        } else {
          const int k0 = c0 + j * 32, dist0 = qpos - k0;
          const int kp = keep - k0;
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            const int dist = dist0 - e;
            const float bv = biased ? bias_s[max(0, min(dist, sat))] : 0.f;
            const bool seen = dist >= 0 && (!windowed || k0 + e >= first || e < kp);
            const float y = soft ? capped(__uint_as_float(v[e])) : fmaf(__uint_as_float(v[e]), scale2, bv);
            const float x = seen ? y : -INFINITY;
            mx[e & 3] = fmaxf(mx[e & 3], x);
            v[e] = __float_as_uint(x);
          }
          tmem_st_32x32(s_addr + j * 32, v);
          cmax = fmaxf(cmax, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])));
        }
      }
      tmem_st_wait();
      // move the reference where the maximum has outgrown it
      const bool move = cmax > m_ref + PF_SLACK || (m_ref == -INFINITY && cmax > -INFINITY);
      if (__any_sync(0xffffffffu, move)) {
        const float m_new = move ? cmax : m_ref;
        const float alpha = move ? exp2f(m_ref - m_new) : 1.f;  // exp2(-inf) = 0: nothing seen before
        l_run *= alpha;
        m_ref = m_new;
        if (c > 0) {  // S of this chunk was issued after the previous P.V had completed: O is at rest
#pragma unroll 1
          for (int j = 0; j * 32 < p.Dv; ++j) {
            uint32_t v[32];
            tmem_ld_32x32(o_addr + j * 32, v);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) v[e] = __float_as_uint(__uint_as_float(v[e]) * alpha);
            tmem_st_32x32(o_addr + j * 32, v);
          }
        }
      }
      const float ref = m_ref == -INFINITY ? 0.f : m_ref;
      // pass 2: weights, hi and lo terms over the scores they came from
      float ls[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
      for (int j = 0; j < GROUPS; ++j) {
        uint32_t v[32];
        if (none >> j & 1) {
#pragma unroll
          for (int e = 0; e < 32; ++e) v[e] = 0;
        } else {
          const bool pl = plain >> j & 1;
          const float a = pl && !soft ? scale2 : 1.f, bb = pl ? bias_far - ref : -ref;
          tmem_ld_32x32(s_addr + j * 32, v);
          tmem_ld_wait();
          if (small >> j & 1) {
#pragma unroll
            for (int e = 0; e < 32; ++e) v[e] = __float_as_uint(capped_small(__uint_as_float(v[e])));
          } else if (pl && soft) {
#pragma unroll
            for (int e = 0; e < 32; ++e) v[e] = __float_as_uint(capped(__uint_as_float(v[e])));
          }
          uint32_t w[32];
#pragma unroll
          for (int e = 0; e < 32; e += 2) {
            const float p0 = exp2f(fmaf(__uint_as_float(v[e]), a, bb)), p1 = exp2f(fmaf(__uint_as_float(v[e + 1]), a, bb));
            ls[e >> 1 & 3] += p0 + p1;
            const uint32_t h = pack_bf16x2(p0, p1);
            w[e >> 1] = h;
            w[16 + (e >> 1)] = pack_bf16x2(p0 - __uint_as_float(h << 16), p1 - __uint_as_float(h & 0xffff0000u));
          }
#pragma unroll
          for (int e = 0; e < 32; ++e) v[e] = w[e];
        }
        tmem_st_32x32(s_addr + j * 32, v);
      }
      l_run += (ls[0] + ls[1]) + (ls[2] + ls[3]);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    if (ok && (*abort_flag || !mbar_wait(o_full, (n_chunks - 1) & 1))) {
      report_error(p.status, ERR_WAIT_TMEM_FULL, 1000);
      *abort_flag = 1;
      ok = false;
    }
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
      float inv = l_run > 0.f ? 1.f / l_run : 0.f;
      if (p.gate && p.gate_w == 1 && r0 + r < n_q)  // one number for the head
        inv = __fdividef(inv, 1.f + __expf(-__bfloat162float(p.gate[(long long)(q_first + r0 + r) * p.gate_stride + hq])));
      const __nv_bfloat16* gate =
          p.gate && p.gate_w != 1 ? p.gate + (long long)(q_first + r0 + r) * p.gate_stride + (long long)hq * p.Dv : nullptr;
      __nv_bfloat16* dst = p.out + (long long)(q_first + r0 + r) * p.out_stride + (long long)hq * p.Dv;
#pragma unroll 1
      for (int j = 0; j * 32 < p.Dv; ++j) {
        uint32_t v[32];
        tmem_ld_32x32(o_addr + j * 32, v);
        tmem_ld_wait();
        if (r0 + r < n_q) {
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            if (j * 32 + k * 8 < p.Dv) {
              float f[8];
#pragma unroll
              for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(v[8 * k + e]) * inv;
              if (gate) {
                const uint4 raw = *reinterpret_cast<const uint4*>(gate + j * 32 + k * 8);
                const uint32_t g[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
                for (int e = 0; e < 8; ++e)
                  f[e] = __fdividef(f[e], 1.f + __expf(-__uint_as_float(e & 1 ? g[e >> 1] & 0xffff0000u : g[e >> 1] << 16)));
              }
              *reinterpret_cast<uint4*>(dst + j * 32 + k * 8) = make_uint4(
                  pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
            }
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 256);
  }
}

}  // namespace vb

using namespace vb;

extern "C" int vb_paged_flash_supported(int Hq, int Hk, int D, int Dv, int block_size, int bias_len) {
  return Hk > 0 && Hq % Hk == 0 && D >= 8 && D <= 128 && Dv >= 8 && Dv <= 128 && (D & 7) == 0 && (Dv & 7) == 0 &&
         block_size >= 8 && block_size <= 128 && 128 % block_size == 0 && bias_len <= PF_MAX_BIAS;
}

// q [T, Hq, D] bf16 (token stride q_stride elements, a multiple of 8); caches [num_blocks, Hk, block_size, D | Dv]; the
// queries of sequence b are the last cu_q[b + 1] - cu_q[b] of its seq_lens[b] positions; out [T, Hq * Dv]. Window (with kept
// first keys) or chunk; bias or softcap; sink [Hq] fp32 and gate [T, Hq * Dv] (gate_w 1: [T, Hq]) bf16 or null; shift [Hq] fp32
// (without bias, softcap and sink) with r1, r2 [Hq] or null: sigmoid weights.
extern "C" int vb_paged_flash(const void* q, long long q_stride, const void* kc, const void* vc, int num_blocks,
                              const int* block_table, int max_blocks, const int* cu_q, const int* seq_lens, int T, int B,
                              int max_q, int Hq, int Hk, int D, int Dv, int block_size, float scale, int window,
                              int keep_first, int chunk, const float* bias, int bias_len, float softcap, const float* sink,
                              const float* shift, const float* r1, const float* r2, const void* gate, long long gate_stride,
                              int gate_w, void* out, long long out_stride, int* status, cudaStream_t stream) {
  if (B <= 0 || T <= 0 || max_q <= 0) return 0;
  if (!vb_paged_flash_supported(Hq, Hk, D, Dv, block_size, bias_len) || (q_stride & 7) || (out_stride & 7) || B > 65535 ||
      (bias != nullptr && bias_len <= 0) || (window > 0 && chunk > 0) || (softcap > 0.f && bias != nullptr) ||
      (gate != nullptr && gate_w != 1 && ((gate_stride & 7) || (reinterpret_cast<uintptr_t>(gate) & 15))) ||
      (shift && (bias || sink || softcap > 0.f)) || (r1 && (!shift || !r2)))
    return -3;
  CUtensorMap tmQ, tmK, tmV;
  int rc = vb_make_tmap_3d(&tmQ, q, 2, (uint64_t)D, (uint64_t)Hq, (uint64_t)T, (uint64_t)D * 2, (uint64_t)q_stride * 2, 64, 1,
                           PF_M);
  if (rc) return rc;
  const uint64_t rows = (uint64_t)num_blocks * Hk * block_size;
  rc = vb_make_tmap_2d(&tmK, kc, 2, (uint64_t)D, rows, (uint64_t)D * 2, 64, block_size);
  if (rc) return rc;
  rc = vb_make_tmap_2d(&tmV, vc, 2, (uint64_t)Dv, rows, (uint64_t)Dv * 2, 64, block_size);
  if (rc) return rc;
  const int smem = PfCfg<false>::BIAS_OFF + (shift ? 2 * PF_TAB * 4 : bias ? bias_len * 4 : 0) + 1024;
  static bool attr_set = false;
  if (!attr_set) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(paged_flash_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       PfCfg<false>::BIAS_OFF + PF_MAX_BIAS * 4 + 1024));
    VB_CUDA_CHECK(cudaFuncSetAttribute(paged_flash_kernel<false, true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       PfCfg<false>::BIAS_OFF + 2 * PF_TAB * 4 + 1024));
    attr_set = true;
  }
  PagedFlashParams p{};
  p.cu_q = cu_q; p.seq_lens = seq_lens; p.block_table = block_table; p.bias = bias;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.out_stride = out_stride;
  p.max_blocks = max_blocks; p.Hq = Hq; p.Hk = Hk; p.D = D; p.Dv = Dv; p.block_size = block_size;
  p.window = window; p.keep_first = keep_first; p.chunk = chunk; p.bias_len = bias_len;
  p.max_qblocks = (max_q + PF_M - 1) / PF_M;
  p.scale = scale; p.softcap = softcap; p.sink = sink;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate);
  p.gate_stride = gate_stride;
  p.gate_w = gate_w;
  p.shift = shift; p.r1 = r1; p.r2 = r2;
  p.status = status;
  const dim3 grid(p.max_qblocks, Hq, B);
  cudaError_t e = shift ? vb_launch_pdl(paged_flash_kernel<false, true>, grid, dim3(PF_THREADS), (size_t)smem, stream, 1, tmQ, tmK,
                                        tmV, tmQ, tmK, p)
                        : vb_launch_pdl(paged_flash_kernel<false>, grid, dim3(PF_THREADS), (size_t)smem, stream, 1, tmQ, tmK,
                                        tmV, tmQ, tmK, p);
  vb_count_launch();
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

extern "C" int vb_latent_flash_supported(int H, int dim, int rot, int vdim, int rank) {
  return H > 0 && dim >= 8 && dim <= 128 && rot >= 8 && vdim >= 8 && vdim <= 128 && (dim & 7) == 0 && (rot & 7) == 0 &&
         (vdim & 7) == 0 && (rank & 7) == 0 && (dim + 63) / 64 + (rot + 63) / 64 <= PfCfg<true>::HALVES;
}

// q [T, H, dim + rot] bf16 (token stride q_stride); the contexts' rotated key parts [N, rot] (row stride rot_stride) and
// expanded rows [N, H * dim keys | H * vdim values] (row stride kv_stride), sequence b from row ctx_cu[b]; its queries are
// the rows cu_q[b] .. cu_q[b + 1] - 1 of q, the last positions of its context. out, window, sink as above; gate_w: numbers of the
// gate per head, vdim or 1.
extern "C" int vb_latent_flash(const void* q, long long q_stride, int T, const void* rot_keys, long long rot_stride,
                               const void* kv, long long kv_stride, int N, const int* cu_q, const int* ctx_cu, int B, int max_q,
                               int H, int dim, int rot, int vdim, float scale, int window, const float* sink, const void* gate,
                               long long gate_stride, int gate_w, void* out, long long out_stride, int* status,
                               cudaStream_t stream) {
  if (B <= 0 || T <= 0 || max_q <= 0 || N <= 0) return 0;
  if (!vb_latent_flash_supported(H, dim, rot, vdim, 8) || (q_stride & 7) || (rot_stride & 7) || (kv_stride & 7) ||
      (out_stride & 7) || B > 65535 || (gate != nullptr && gate_w != 1 && gate_w != vdim) ||
      (gate != nullptr && gate_w != 1 && ((gate_stride & 7) || (reinterpret_cast<uintptr_t>(gate) & 15))))
    return -3;
  const __nv_bfloat16 *qb = reinterpret_cast<const __nv_bfloat16*>(q), *kb = reinterpret_cast<const __nv_bfloat16*>(kv);
  const uint64_t head = (uint64_t)(dim + rot) * 2, row = (uint64_t)kv_stride * 2;
  constexpr int KEYS = PfCfg<true>::N;
  CUtensorMap tmQ, tmQr, tmK, tmKr, tmV;
  int rc = vb_make_tmap_3d(&tmQ, qb, 2, dim, H, T, head, (uint64_t)q_stride * 2, 64, 1, PF_M);
  if (!rc) rc = vb_make_tmap_3d(&tmQr, qb + dim, 2, rot, H, T, head, (uint64_t)q_stride * 2, 64, 1, PF_M);
  if (!rc) rc = vb_make_tmap_3d(&tmK, kb, 2, dim, H, N, (uint64_t)dim * 2, row, 64, 1, KEYS);
  if (!rc) rc = vb_make_tmap_3d(&tmV, kb + (long long)H * dim, 2, vdim, H, N, (uint64_t)vdim * 2, row, 64, 1, KEYS);
  if (!rc) rc = vb_make_tmap_2d(&tmKr, rot_keys, 2, rot, N, (uint64_t)rot_stride * 2, 64, KEYS);
  if (rc) return rc;
  const int smem = PfCfg<true>::BIAS_OFF + 1024;
  static bool attr_set = false;
  if (!attr_set) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(paged_flash_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr_set = true;
  }
  PagedFlashParams p{};
  p.cu_q = cu_q; p.ctx_cu = ctx_cu;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.out_stride = out_stride;
  p.Hq = H; p.Hk = H; p.D = dim; p.rot = rot; p.Dv = vdim;
  p.max_qblocks = (max_q + PF_M - 1) / PF_M;
  p.scale = scale; p.window = window; p.sink = sink;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate);
  p.gate_stride = gate_stride;
  p.gate_w = gate_w;
  p.status = status;
  const dim3 grid(p.max_qblocks, H, B);
  cudaError_t e = vb_launch_pdl(paged_flash_kernel<true>, grid, dim3(PF_THREADS), (size_t)smem, stream, 1, tmQ, tmK, tmV, tmQr,
                                tmKr, p);
  vb_count_launch();
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
