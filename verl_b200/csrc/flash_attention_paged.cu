// Prefill attention of layer-list decoders on tcgen05: ragged queries over the paged KV cache, with a sliding window,
// kept first keys and a per-distance bias. Head sizes up to 128 (multiples of 8), bf16.
//
// One CTA per (sequence, query head, block of 128 queries). The CTA walks the 128-key chunks that some row of the block
// may see: those of the kept first keys, then those of the window. Per chunk:
//     S[128 q x 128 keys] = Q . K^T                       (tcgen05.mma, accumulator in TMEM)
//     P = exp(S * scale + bias[distance] - rowmax)        (thread = query row)
//     O_c[128 q x Dv]     = P . V                         (A operand = P in TMEM)
// The weights stay close to fp32: P is split into two bf16 terms (P = hi + lo) that are written over the columns of S
// they came from, and both are multiplied with V. The running output lives in registers (flash rescale).
// K / V pages arrive by per-CTA TMA loads through a ring of 32 KB slots; columns past a head's size are filled with zeros
// by TMA, keys past the sequence or outside the mask get weight zero.
// Every wait is bounded; on expiry the status word is set and the CTA leaves through its teardown.
#include "common.cuh"
#include "host_utils.h"

namespace vb {

constexpr int PF_M = 128, PF_N = 128;             // queries per CTA, keys per chunk
constexpr int PF_TILE = 128 * 128 * 2;            // 32 KB: two 64-column halves of 16 KB
constexpr int PF_SLOTS = 5;
constexpr int PF_THREADS = 192;
constexpr int PF_RING_OFF = PF_TILE;              // Q first
constexpr int PF_BAR_OFF = PF_RING_OFF + PF_SLOTS * PF_TILE;
constexpr int PF_BIAS_OFF = PF_BAR_OFF + 20 * 8 + 32;
constexpr int PF_MAX_BIAS = 6144;                 // distances staged in shared memory

struct PagedFlashParams {
  const int* cu_q;         // [B + 1]
  const int* seq_lens;     // [B]
  const int* block_table;  // [B, max_blocks]
  const float* bias;       // [Hq, bias_len] or null
  __nv_bfloat16* out;      // [T, out_stride]
  long long out_stride;
  int max_blocks, Hq, Hk, D, Dv, block_size, window, keep_first, bias_len, max_qblocks;
  float scale;
  int* status;
};

// exp2 of the scaled scores: scale and bias are multiplied by log2(e) up front
constexpr float LOG2E = 1.4426950408889634f;

__global__ void __launch_bounds__(PF_THREADS, 1)
paged_flash_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                   const __grid_constant__ CUtensorMap tmV, const PagedFlashParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;
  uint8_t* ring = smem + PF_RING_OFF;
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + PF_BAR_OFF);
  uint64_t* empty = full + PF_SLOTS;
  uint64_t* s_full = empty + PF_SLOTS;
  uint64_t* p_ready = s_full + 2;
  uint64_t* o_full = p_ready + 2;
  uint64_t* q_full = o_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* bias_s = reinterpret_cast<float*>(smem + PF_BIAS_OFF);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.z, hq = blockIdx.y;
  pdl_wait();
  const int q_first = p.cu_q[b], n_q = p.cu_q[b + 1] - q_first;
  const int r0 = (p.max_qblocks - 1 - (int)blockIdx.x) * PF_M;  // late blocks (most keys) first
  if (r0 >= n_q) return;  // uniform for the CTA, before any barrier or allocation
  const int hk = hq / (p.Hq / p.Hk);
  const int seq_len = p.seq_lens[b];
  const int pos0 = seq_len - n_q + r0;                     // position of row 0
  const int pos1 = min(pos0 + PF_M, seq_len) - 1;          // last real row
  const bool windowed = p.window > 0;
  const int keep = windowed ? p.keep_first : 0;
  // chunks to visit: [0, keep_chunks) and [win_chunk, last_chunk]
  const int last_chunk = pos1 / PF_N;
  const int keep_chunks = min((keep + PF_N - 1) / PF_N, last_chunk + 1);
  const int win_chunk = max(windowed ? max(pos0 - p.window + 1, 0) / PF_N : 0, keep_chunks);
  const int n_chunks = keep_chunks + max(last_chunk + 1 - win_chunk, 0);
  auto chunk_at = [&](int c) { return c < keep_chunks ? c : win_chunk + c - keep_chunks; };

  if (tid == 0) {
    for (int s = 0; s < PF_SLOTS; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_ready[i], 4);
      mbar_init(&o_full[i], 1);
    }
    mbar_init(q_full, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  if (p.bias != nullptr)
    for (int i = tid; i < p.bias_len; i += PF_THREADS) bias_s[i] = p.bias[(long long)hq * p.bias_len + i] * LOG2E;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_trigger();  // TMEM is held: a dependent kernel may take what is left
  const int k_halves = p.D > 64 ? 2 : 1, v_halves = p.Dv > 64 ? 2 : 1;

  if (warp == 4) {
    // ------------------------------- TMA producer -------------------------------
    if (lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      mbar_arrive_expect_tx(q_full, k_halves * 16384);
      for (int x = 0; x < k_halves; ++x) tma_load_3d(q_s + x * 16384, &tmQ, q_full, x * 64, hq, q_first + r0);
      const int* bt = p.block_table + (long long)b * p.max_blocks;
      const int ppc = PF_N / p.block_size, n_pages = (seq_len + p.block_size - 1) / p.block_size;
      for (int t = 0; t < 2 * n_chunks; ++t) {
        const int s = t % PF_SLOTS;
        if (*abort_flag || !mbar_wait(&empty[s], ((t / PF_SLOTS) & 1) ^ 1)) {
          report_error(p.status, ERR_WAIT_EMPTY, t);
          *abort_flag = 1;
          break;
        }
        const int halves = (t & 1) ? v_halves : k_halves;
        mbar_arrive_expect_tx(&full[s], halves * 16384);
        uint8_t* dst = ring + s * PF_TILE;
        const CUtensorMap* tm = (t & 1) ? &tmV : &tmK;
        const int page0 = chunk_at(t >> 1) * ppc;
        for (int pg = 0; pg < ppc; ++pg) {
          // pages past the end re-read the last page: finite data, weight zero
          const int row = (bt[min(page0 + pg, n_pages - 1)] * p.Hk + hk) * p.block_size;
          for (int x = 0; x < halves; ++x)
            tma_load_2d(dst + x * 16384 + pg * p.block_size * 128, tm, &full[s], x * 64, row);
        }
      }
    }
  } else if (warp == 5) {
    // -------------------------------- MMA issuer --------------------------------
    if (lane == 0) {
      const uint32_t idesc_qk = umma_idesc(1, 1, 0, 0, PF_M, PF_N);
      const uint32_t idesc_pv = umma_idesc(1, 1, 0, 1, PF_M, (uint32_t)((p.Dv + 15) / 16 * 16));
      const uint32_t q_addr = smem_u32(q_s);
      const int k_steps = (p.D + 15) / 16;
      bool ok = !*abort_flag && mbar_wait(q_full, 0);
      if (!ok) {
        report_error(p.status, ERR_WAIT_FULL, 9000);
        *abort_flag = 1;
      }
      auto issue_qk = [&](int c) -> bool {
        const int t = 2 * c, s = t % PF_SLOTS;
        // the buffer holds P of chunk c - 2 until its P.V has completed
        if (c >= 2 && (*abort_flag || !mbar_wait(&o_full[c & 1], ((c - 2) >> 1) & 1))) {
          report_error(p.status, ERR_WAIT_TMEM_EMPTY, 2000 + c);
          *abort_flag = 1;
          return false;
        }
        if (*abort_flag || !mbar_wait(&full[s], (t / PF_SLOTS) & 1)) {
          report_error(p.status, ERR_WAIT_FULL, t);
          *abort_flag = 1;
          return false;
        }
        tc_fence_after();
        const uint32_t k_addr = smem_u32(ring + s * PF_TILE);
        for (int k = 0; k < k_steps; ++k) {
          const uint32_t off = (k >> 2) * 16384 + (k & 3) * 32;
          tc_mma_f16(tmem_base + (c & 1) * PF_N, umma_smem_desc(q_addr + off, 16, 1024),
                     umma_smem_desc(k_addr + off, 16, 1024), idesc_qk, k != 0);
        }
        tc_commit(&s_full[c & 1]);
        tc_commit(&empty[s]);
        return true;
      };
      if (ok) ok = issue_qk(0);
      for (int c = 0; ok && c < n_chunks; ++c) {
        if (c + 1 < n_chunks) ok = issue_qk(c + 1);
        if (!ok) break;
        const int t = 2 * c + 1, s = t % PF_SLOTS;
        if (*abort_flag || !mbar_wait(&full[s], (t / PF_SLOTS) & 1)) {
          report_error(p.status, ERR_WAIT_FULL, t);
          *abort_flag = 1;
          break;
        }
        if (*abort_flag || !mbar_wait(&p_ready[c & 1], (c >> 1) & 1)) {
          report_error(p.status, ERR_WAIT_TMEM_EMPTY, c);
          *abort_flag = 1;
          break;
        }
        tc_fence_after();
        const uint32_t v_addr = smem_u32(ring + s * PF_TILE);
        const uint32_t p_tmem = tmem_base + (c & 1) * PF_N, d_tmem = tmem_base + 256 + (c & 1) * 128;
#pragma unroll
        for (int k = 0; k < PF_N / 16; ++k) {
          const uint64_t bv = umma_smem_desc(v_addr + k * 2048, 16384, 1024);
          const uint32_t a = p_tmem + (k >> 1) * 32 + (k & 1) * 8;  // per 32 keys: 16 columns of hi, 16 of lo
          tc_mma_f16_ta(d_tmem, a, bv, idesc_pv, k != 0);
          tc_mma_f16_ta(d_tmem, a + 16, bv, idesc_pv, 1);
        }
        tc_commit(&o_full[c & 1]);
        tc_commit(&empty[s]);
      }
    }
  } else {
    // ----------------------- softmax + accumulation (128 threads, thread = query row) -----------------------
    const int r = tid, qpos = pos0 + r;
    const uint32_t lane_base = ((uint32_t)(warp * 32)) << 16;
    const float scale2 = p.scale * LOG2E;
    const int sat = p.bias_len - 1;
    const float bias_far = p.bias != nullptr ? bias_s[sat] : 0.f;
    float o_acc[128];
#pragma unroll
    for (int i = 0; i < 128; ++i) o_acc[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    float alpha_cur = 1.f, alpha_nxt = 1.f;
    bool ok = true;

    auto softmax_chunk = [&](int c) -> float {
      const int i = c & 1;
      if (*abort_flag || !mbar_wait(&s_full[i], (c >> 1) & 1)) {
        report_error(p.status, ERR_WAIT_TMEM_FULL, c);
        *abort_flag = 1;
        ok = false;
      }
      const int c0 = chunk_at(c) * PF_N;
      // key c0 + e is visible iff e < lim and (e >= wlo or e < kp)
      const int lim = qpos - c0 + 1;
      const int wlo = windowed ? qpos - p.window + 1 - c0 : -1;
      const int kp = keep - c0;
      const bool all = lim >= PF_N && (wlo <= 0 || kp >= PF_N);
      const bool far = p.bias == nullptr || qpos - (c0 + PF_N - 1) >= sat;  // every distance is past the table
      const bool plain = __all_sync(0xffffffffu, all && far);
      const uint32_t s_addr = tmem_base + lane_base + i * PF_N;
      // scaled, biased, masked score of element e
      auto score = [&](uint32_t raw, int e) -> float {
        float x = fmaf(__uint_as_float(raw), scale2, bias_far);
        if (!plain) {
          if (p.bias != nullptr) x = fmaf(__uint_as_float(raw), scale2, bias_s[max(0, min(qpos - c0 - e, sat))]);
          if (!(e < lim && (e >= wlo || e < kp))) x = -INFINITY;
        }
        return x;
      };
      float cmax = -INFINITY;
      if (ok) {
        tc_fence_after();
#pragma unroll 1
        for (int j = 0; j < PF_N / 32; ++j) {
          uint32_t v[32];
          tmem_ld_32x32(s_addr + j * 32, v);
          tmem_ld_wait();
          if (plain) {
            // scale2 may be negative: take both ends
            float hi = __uint_as_float(v[0]), lo = hi;
#pragma unroll
            for (int e = 1; e < 32; ++e) {
              hi = fmaxf(hi, __uint_as_float(v[e]));
              lo = fminf(lo, __uint_as_float(v[e]));
            }
            cmax = fmaxf(cmax, fmaf(scale2 >= 0.f ? hi : lo, scale2, bias_far));
          } else {
#pragma unroll
            for (int e = 0; e < 32; ++e) cmax = fmaxf(cmax, score(v[e], j * 32 + e));
          }
        }
      }
      const float m_new = fmaxf(m_run, cmax);
      const float m_ref = (m_new == -INFINITY) ? 0.f : m_new;  // no visible key so far: avoid inf - inf
      const float alpha = exp2f(m_run - m_ref);
      float lsum = 0.f;
      if (ok) {
#pragma unroll 1
        for (int j = 0; j < PF_N / 32; ++j) {
          uint32_t v[32], w[32];
          tmem_ld_32x32(s_addr + j * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; e += 2) {
            const float p0 = exp2f(score(v[e], j * 32 + e) - m_ref);
            const float p1 = exp2f(score(v[e + 1], j * 32 + e + 1) - m_ref);
            lsum += p0 + p1;
            const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
            const float2 hf = __bfloat1622float2(h);
            w[e >> 1] = *reinterpret_cast<const uint32_t*>(&h);
            w[16 + (e >> 1)] = pack_bf16x2(p0 - hf.x, p1 - hf.y);
          }
          tmem_st_32x32(s_addr + j * 32, w);
        }
        tmem_st_wait();
      }
      m_run = m_new;
      l_run = l_run * alpha + lsum;
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[i]);
      return alpha;
    };

    alpha_cur = softmax_chunk(0);
    for (int c = 0; c < n_chunks; ++c) {
      const int i = c & 1;
      if (c + 1 < n_chunks) alpha_nxt = softmax_chunk(c + 1);
      if (ok && (*abort_flag || !mbar_wait(&o_full[i], (c >> 1) & 1))) {
        report_error(p.status, ERR_WAIT_TMEM_FULL, 1000 + c);
        *abort_flag = 1;
        ok = false;
      }
      // the lanes of a warp share its TMEM loads: they stop together
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        tc_fence_after();
        const uint32_t o_addr = tmem_base + lane_base + 256 + i * 128;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (j * 32 < p.Dv) {
            uint32_t v[32];
            tmem_ld_32x32(o_addr + j * 32, v);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) o_acc[j * 32 + e] = o_acc[j * 32 + e] * alpha_cur + __uint_as_float(v[e]);
          }
        }
      }
      alpha_cur = alpha_nxt;
      if (!ok) break;
    }
    if (ok && r0 + r < n_q) {
      const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
      __nv_bfloat16* dst = p.out + (long long)(q_first + r0 + r) * p.out_stride + (long long)hq * p.Dv;
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        if (j * 8 < p.Dv) {
          uint4 w;
          w.x = pack_bf16x2(o_acc[8 * j] * inv, o_acc[8 * j + 1] * inv);
          w.y = pack_bf16x2(o_acc[8 * j + 2] * inv, o_acc[8 * j + 3] * inv);
          w.z = pack_bf16x2(o_acc[8 * j + 4] * inv, o_acc[8 * j + 5] * inv);
          w.w = pack_bf16x2(o_acc[8 * j + 6] * inv, o_acc[8 * j + 7] * inv);
          reinterpret_cast<uint4*>(dst)[j] = w;
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

}  // namespace vb

using namespace vb;

extern "C" int vb_paged_flash_supported(int Hq, int Hk, int D, int Dv, int block_size, int bias_len) {
  return Hk > 0 && Hq % Hk == 0 && D >= 8 && D <= 128 && Dv >= 8 && Dv <= 128 && (D & 7) == 0 && (Dv & 7) == 0 &&
         block_size >= 8 && block_size <= 128 && PF_N % block_size == 0 && bias_len <= PF_MAX_BIAS;
}

// q [T, Hq, D] bf16 (token stride q_stride elements, a multiple of 8); caches [num_blocks, Hk, block_size, D | Dv]; the
// queries of sequence b are the last cu_q[b + 1] - cu_q[b] of its seq_lens[b] positions; out [T, Hq * Dv].
extern "C" int vb_paged_flash(const void* q, long long q_stride, const void* kc, const void* vc, int num_blocks,
                              const int* block_table, int max_blocks, const int* cu_q, const int* seq_lens, int T, int B,
                              int max_q, int Hq, int Hk, int D, int Dv, int block_size, float scale, int window,
                              int keep_first, const float* bias, int bias_len, void* out, long long out_stride, int* status,
                              cudaStream_t stream) {
  if (B <= 0 || T <= 0 || max_q <= 0) return 0;
  if (!vb_paged_flash_supported(Hq, Hk, D, Dv, block_size, bias_len) || (q_stride & 7) || (out_stride & 7) || B > 65535 ||
      (bias != nullptr && bias_len <= 0))
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
  const int smem = PF_BIAS_OFF + (bias ? bias_len * 4 : 0) + 1024;
  static bool attr_set = false;
  if (!attr_set) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(paged_flash_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       PF_BIAS_OFF + PF_MAX_BIAS * 4 + 1024));
    attr_set = true;
  }
  PagedFlashParams p{cu_q, seq_lens, block_table, bias, reinterpret_cast<__nv_bfloat16*>(out), out_stride, max_blocks, Hq, Hk, D,
                     Dv, block_size, window, keep_first, bias_len, (max_q + PF_M - 1) / PF_M, scale, status};
  const dim3 grid(p.max_qblocks, Hq, B);
  cudaError_t e = vb_launch_pdl(paged_flash_kernel, grid, dim3(PF_THREADS), (size_t)smem, stream, 1, tmQ, tmK, tmV, p);
  vb_count_launch();
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}
