// Latent attention in the latent space on tcgen05 (short portions and decoding), bf16.
//
// head_gemm: out[t, h, :] = a[t, h, :] . B_h for every head h of ragged token rows, the up projections of latent attention
// applied to queries (and to weighted sums, times the sigmoid of an output gate). One CTA per (head, 128 rows, 64 columns).
//
// latent_decode: paged attention whose one "key head" is the row of the cache itself: `width` numbers (a multiple of 64), the
// first `rank` of them being the value as well, so a row is read once. One CTA per (query row, group of up to 32 heads,
// split of the keys). Work is transposed as in paged_attention_tc.cu, 64 keys at a time:
//     S^T[keys x heads]  = C[64 keys x width] . Q^T          (M = keys, N = heads)
//     O^T[rank x heads] += C^T[rank x 64 keys] . P           (M = 128 dims per block, N = 2 x heads)
// A stage holds 64 whole rows and serves both products; a second one loads meanwhile. A row is wide, so one copy takes all
// 64-column parts of eight rows: a stage is [8 groups][parts][8 rows x 128 bytes], and both products address it through the
// strides of their descriptors. (The tensor core reads the first operand of these narrow products slowly enough for its rows
// to count: M = 64 for the scores. An accumulator of 64 rows lies in the first 16 lanes of each warp's 32.)
// P is two bf16 terms (hi in the columns of the heads, lo behind them), so that the weights stay close to fp32; both land in
// accumulators of their own and are added at the end. O^T accumulates in TMEM over all keys: a head's reference only moves
// when its maximum has grown by more than 2^8, and every thread keeps the sum of its own keys' weights until the end.
// Every wait is bounded; on expiry the status word is set and the CTA leaves through its teardown.
#include "common.cuh"
#include "host_utils.h"

namespace vb {

// byte offset of element (row r, col k) inside a K-major, 128-byte-swizzled operand of `rows` rows whose k extent is split
// in 64-element blocks of rows * 128 bytes
__device__ __forceinline__ uint32_t sw128_at(int r, int k, int rows) {
  const int kb = k >> 6, c16 = (k & 63) >> 3;
  return (uint32_t)(kb * rows * 128 + (r >> 3) * 1024 + (r & 7) * 128 + ((c16 ^ (r & 7)) << 4) + (k & 7) * 2);
}

// ------------------------------------------------------------------------------------------------ per-head products
constexpr int HG_STAGES = 4, HG_A = 128 * 128, HG_B = 64 * 128, HG_STAGE = HG_A + HG_B, HG_THREADS = 192;
constexpr int HG_BAR_OFF = HG_STAGES * HG_STAGE, HG_SMEM = HG_BAR_OFF + (2 * HG_STAGES + 1) * 8 + 16 + 1024;

struct HeadGemmParams {
  const __nv_bfloat16* a;
  long long a_t, a_h;
  __nv_bfloat16* out;
  long long o_t, o_h;
  const __nv_bfloat16* gate;  // [T, H * N] (gate_w 1: [T, H]) or null
  long long gate_stride;
  int gate_w, T, K, N, tail, width, b_mn;
  int* status;
};

__global__ void __launch_bounds__(HG_THREADS, 2)
head_gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const HeadGemmParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + HG_BAR_OFF);
  uint64_t *empty = full + HG_STAGES, *done = empty + HG_STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int tid = threadIdx.x, warp = tid >> 5;
  const int h = blockIdx.y, m0 = blockIdx.z * 128, n0 = blockIdx.x * 64;
  const int steps = (p.K + 63) / 64;

  if (tid == 0) {
    for (int s = 0; s < 2 * HG_STAGES + 1; ++s) mbar_init(&full[s], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, 64);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_trigger();  // TMEM is held: a dependent kernel may take what is left
  pdl_wait();

  if (warp == 4) {
    if (elect_one()) {
      int k = 0;
      for (; k < steps; ++k) {
        const int s = k % HG_STAGES;
        if (*abort_flag || !mbar_wait(&empty[s], ((k / HG_STAGES) & 1) ^ 1)) {
          report_error(p.status, ERR_WAIT_EMPTY, k);
          *abort_flag = 1;
          break;
        }
        mbar_arrive_expect_tx(&full[s], HG_STAGE);
        uint8_t* dst = smem + s * HG_STAGE;
        tma_load_3d(dst, &tmA, &full[s], k * 64, h, m0);
        if (p.b_mn) tma_load_3d(dst + HG_A, &tmB, &full[s], n0, k * 64, h);
        else tma_load_3d(dst + HG_A, &tmB, &full[s], k * 64, n0, h);
      }
      for (int i = max(k - HG_STAGES, 0); i < k; ++i) mbar_wait(&full[i % HG_STAGES], (i / HG_STAGES) & 1);  // none in flight
    }
  } else if (warp == 5) {
    if (elect_one()) {
      const uint32_t idesc = umma_idesc(1, 1, 0, p.b_mn ? 1 : 0, 128, 64), base = smem_u32(smem);
      for (int k = 0; k < steps; ++k) {
        const int s = k % HG_STAGES;
        if (*abort_flag || !mbar_wait(&full[s], (k / HG_STAGES) & 1)) {
          report_error(p.status, ERR_WAIT_FULL, k);
          *abort_flag = 1;
          break;
        }
        tc_fence_after();
        const uint32_t a = base + s * HG_STAGE, b = a + HG_A;
#pragma unroll
        for (int i = 0; i < 4; ++i)
          tc_mma_f16(tmem, umma_smem_desc(a + i * 32, 16, 1024),
                     p.b_mn ? umma_smem_desc(b + i * 2048, HG_B, 1024) : umma_smem_desc(b + i * 32, 16, 1024), idesc,
                     k != 0 || i != 0);
        tc_commit(&empty[s]);
        if (k == steps - 1) tc_commit(done);
      }
    }
  } else {
    bool ok = !*abort_flag && mbar_wait(done, 0);
    if (!ok) {
      report_error(p.status, ERR_WAIT_TMEM_FULL, 1);
      *abort_flag = 1;
    }
    ok = __all_sync(0xffffffffu, ok);  // the lanes of a warp share its TMEM accesses: they stop together
    const int t = m0 + tid;
    if (ok) {
      tc_fence_after();
      __nv_bfloat16* dst = p.out + t * p.o_t + h * p.o_h;
      float head_gate = 1.f;
      if (p.gate && p.gate_w == 1 && t < p.T)
        head_gate = __fdividef(1.f, 1.f + __expf(-__bfloat162float(p.gate[t * p.gate_stride + h])));
#pragma unroll 1
      for (int j = 0; j < 2; ++j) {
        uint32_t v[32];
        tmem_ld_32x32(tmem + (((uint32_t)(warp * 32)) << 16) + j * 32, v);
        tmem_ld_wait();
        if (t < p.T) {
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int n = n0 + j * 32 + c * 8;
            if (n < p.N) {
              float f[8];
#pragma unroll
              for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(v[8 * c + e]) * head_gate;
              if (p.gate && p.gate_w != 1) {
                const uint4 raw = *reinterpret_cast<const uint4*>(p.gate + t * p.gate_stride + (long long)h * p.N + n);
                const uint32_t g[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
                for (int e = 0; e < 8; ++e)
                  f[e] = __fdividef(f[e], 1.f + __expf(-__uint_as_float(e & 1 ? g[e >> 1] & 0xffff0000u : g[e >> 1] << 16)));
              }
              *reinterpret_cast<uint4*>(dst + n) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]),
                                                              pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
            }
          }
        }
      }
      // behind the product: copied elements, then zeros
      if (blockIdx.x == 0 && t < p.T) {
        const __nv_bfloat16* src = p.a + t * p.a_t + h * p.a_h + p.K;
        for (int i = p.N; i < p.width; i += 8) {  // all sizes but the tail's are multiples of 8
          if (i + 8 <= p.N + p.tail) *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<const uint4*>(src + i - p.N);
          else
            for (int e = i; e < i + 8; ++e) dst[e] = e < p.N + p.tail ? src[e - p.N] : __float2bfloat16(0.f);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, 64);
  }
}

// ------------------------------------------------------------------------------------------------ attention on latents
constexpr int LD_KEYS = 64, LD_THREADS = 224, LD_MAX_STAGES = 6, LD_MAX_PARTS = 10;
constexpr float LD_SLACK = 8.f;
constexpr float LD_LOG2E = 1.4426950408889634f, LD_LN2 = 0.6931471805599453f;

struct LatentDecodeParams {
  const __nv_bfloat16* q;  // [T, H, width]
  const int *block_table, *cu_q, *seq_lens;
  int max_blocks, T, B, H, width, rank, block_size, window, num_splits, stages;
  float scale;
  const float* sink;       // [H] or null
  __nv_bfloat16* out;      // [T, H, rank]
  float *o_part, *ml_part;
  int* status;
};

// shared memory: stages, Q, two P buffers, barriers, reductions
template <int HB>
struct LdCfg {
  static constexpr int P_BYTES = 2 * HB * 128;
  static constexpr int TMEM = HB == 32 ? 512 : 256;      // S: 2 x HB columns, O: up to 4 x 2 HB
  static constexpr int TAIL = 256 + 2 * HB * 16;
  static __host__ __device__ int stage_bytes(int parts) { return parts * LD_KEYS * 128; }
  static __host__ __device__ int q_bytes(int parts) { return parts * HB * 128; }
  static __host__ __device__ int bytes(int stages, int parts) {
    return stages * stage_bytes(parts) + q_bytes(parts) + 2 * P_BYTES + TAIL + 1024;
  }
};

// barrier of the 128 softmax threads that also combines a predicate
__device__ __forceinline__ bool ld_bar_or(bool pred) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 q, %1, 0;\n\tbarrier.red.or.pred p, 1, 128, q;\n\tselp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(r)
      : "r"((uint32_t)pred)
      : "memory");
  return r != 0;
}
__device__ __forceinline__ void ld_bar() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

template <int HB>
__device__ __forceinline__ void ld_cols(uint32_t addr, uint32_t (&v)[HB]) {
  if constexpr (HB == 32) tmem_ld_32x32(addr, v);
  else tmem_ld_32x16(addr, v);
}

template <int HB>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const LatentDecodeParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int parts = p.width >> 6, v_blocks = (p.rank + 127) / 128, stages = p.stages;
  const int stage_bytes = LdCfg<HB>::stage_bytes(parts);
  uint8_t* q_s = smem + stages * stage_bytes;
  uint8_t* p_s = q_s + LdCfg<HB>::q_bytes(parts);
  uint64_t* full = reinterpret_cast<uint64_t*>(p_s + 2 * LdCfg<HB>::P_BYTES);
  uint64_t *empty = full + LD_MAX_STAGES, *s_full = empty + LD_MAX_STAGES, *p_ready = s_full + 2, *o_full = p_ready + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_full + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float(*red_s)[4] = reinterpret_cast<float(*)[4]>(reinterpret_cast<uint8_t*>(full) + 256);
  float(*sum_s)[4] = red_s + HB;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t = blockIdx.x, h0 = blockIdx.y * HB, split = blockIdx.z;
  const int nh = min(HB, p.H - h0);

  if (tid == 0) {
    for (int s = 0; s < LD_MAX_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_ready[i], 4);
      mbar_init(&o_full[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, LdCfg<HB>::TMEM);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_trigger();  // TMEM is held: a dependent kernel may take what is left
  pdl_wait();     // nothing above reads or writes global memory

  int b = t;
  if (p.T != p.B) {  // sequence of row t
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1;
    }
    b = lo;
  }
  const int len = p.seq_lens[b] - (p.T != p.B ? p.cu_q[b + 1] - 1 - t : 0);  // keys that the row sees
  const int key_lo = p.window > 0 ? max(len - p.window, 0) : 0, c_first = key_lo / LD_KEYS;  // first key that it sees
  const int chunks = (len + LD_KEYS - 1) / LD_KEYS, per_split = (chunks - c_first + p.num_splits - 1) / p.num_splits;
  const int c_begin = c_first + split * per_split, n_chunks = max(min(chunks, c_begin + per_split) - c_begin, 0);
  {
    const __nv_bfloat16* q = p.q + ((long long)t * p.H + h0) * p.width;
    const int per_row = parts * 8;
    for (int i = tid; i < HB * per_row; i += LD_THREADS) {
      const int r = i / per_row, k = (i - r * per_row) * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < nh) v = *reinterpret_cast<const uint4*>(q + (long long)r * p.width + k);
      *reinterpret_cast<uint4*>(q_s + sw128_at(r, k, HB)) = v;
    }
  }
  fence_proxy_async_smem();
  __syncthreads();

  if (warp == 4) {
    // ------------------------------- TMA producer: lane g copies rows 8 g .. 8 g + 7 of a chunk -------------------------------
    if (lane == 0) tma_prefetch_desc(&tmC);
    const int* bt = p.block_table + (long long)b * p.max_blocks;
    const int last_page = (len + p.block_size - 1) / p.block_size - 1;
    // first row of the lane's group; pages past the end re-read the last page: finite data, weight zero
    auto row_of = [&](int c) {
      const int key = (c_begin + c) * LD_KEYS + (lane & 7) * 8, page = key / p.block_size;
      return bt[min(page, last_page)] * p.block_size + key - page * p.block_size;
    };
    int row = n_chunks > 0 ? row_of(0) : 0;
    bool ok = true;
    int issued = 0;
    for (int c = 0; ok && c < n_chunks; ++c) {
      const int s = c % stages, next = c + 1 < n_chunks ? row_of(c + 1) : 0;
      int good = 1;  // lane 0 decides for the warp: the lanes must leave the loop together
      if (lane == 0) {
        good = (!*abort_flag && mbar_wait(&empty[s], ((c / stages) & 1) ^ 1)) ? 1 : 0;
        if (good) {
          mbar_arrive_expect_tx(&full[s], stage_bytes);
        } else {
          report_error(p.status, ERR_WAIT_EMPTY, c);
          *abort_flag = 1;
        }
      }
      ok = __shfl_sync(0xffffffffu, good, 0) != 0;
      if (ok && lane < 8) tma_load_3d(smem + s * stage_bytes + lane * parts * 1024, &tmC, &full[s], 0, row, 0);
      __syncwarp();
      row = next;
      issued += ok;
    }
    // no copy is in flight when the CTA ends, whatever ended it
    for (int i = max(issued - stages, 0); lane == 0 && i < issued; ++i) mbar_wait(&full[i % stages], (i / stages) & 1);
  } else if (warp == 5) {
    // -------------------------------- scores --------------------------------
    // The products are small: issuing them takes longer than running them, so that scores and values have a warp each.
    if (n_chunks > 0 && elect_one()) {
      constexpr uint32_t idesc = umma_idesc(1, 1, 0, 0, LD_KEYS, HB);  // A = rows (K-major), B = Q^T (K-major)
      // descriptors of the first tiles; steps are added in units of 16 bytes
      const uint64_t a0 = umma_smem_desc(smem_u32(smem), 16, parts * 1024), b0 = umma_smem_desc(smem_u32(q_s), 16, 1024);
      for (int c = 0; c < n_chunks; ++c) {
        const int s = c % stages;
        // the rows are there, and the scores of chunk c - 2 have been read
        if (*abort_flag || !mbar_wait(&full[s], (c / stages) & 1) || (c > 1 && !mbar_wait(&p_ready[c & 1], ((c >> 1) - 1) & 1))) {
          report_error(p.status, ERR_WAIT_FULL, c);
          *abort_flag = 1;
          break;
        }
        tc_fence_after();
        const uint64_t a = a0 + (uint64_t)s * (stage_bytes >> 4);
        const uint32_t d = tmem + (c & 1) * HB;
        for (int x = 0; x < parts; ++x) {
#pragma unroll
          for (int k = 0; k < 4; ++k) tc_mma_f16(d, a + x * 64 + 2 * k, b0 + x * (HB * 8) + 2 * k, idesc, x != 0 || k != 0);
        }
        tc_commit(&s_full[c & 1]);
      }
    }
  } else if (warp == 6) {
    // -------------------------------- values --------------------------------
    if (n_chunks > 0 && elect_one()) {
      constexpr uint32_t idesc = umma_idesc(1, 1, 1, 0, 128, 2 * HB);  // A = rows (MN-major), B = P (K-major)
      const uint32_t group = parts * 64;                               // 16-byte units from one group of rows to the next
      const uint64_t a0 = umma_smem_desc(smem_u32(smem), 1024, parts * 1024), b0 = umma_smem_desc(smem_u32(p_s), 16, 1024);
      for (int c = 0; c < n_chunks; ++c) {
        const int s = c % stages;
        if (*abort_flag || !mbar_wait(&p_ready[c & 1], (c >> 1) & 1)) {
          report_error(p.status, ERR_WAIT_TMEM_EMPTY, c);
          *abort_flag = 1;
          break;
        }
        tc_fence_after();
        const uint64_t a = a0 + (uint64_t)s * (stage_bytes >> 4), bp = b0 + (c & 1) * (LdCfg<HB>::P_BYTES >> 4);
        for (int v = 0; v < v_blocks; ++v) {
#pragma unroll
          for (int k = 0; k < LD_KEYS / 16; ++k)  // 16 keys: two groups of rows
            tc_mma_f16(tmem + 2 * HB + v * 2 * HB, a + v * 128 + k * 2 * group, bp + 2 * k, idesc, c != 0 || k != 0);
        }
        tc_commit(&empty[s]);
        tc_commit(&o_full[c & 1]);
      }
    }
  } else {
    // ----------------------- softmax (thread = key), then output (thread = dim) -----------------------
    const uint32_t lanes = ((uint32_t)(warp * 32)) << 16, s_addr = tmem + lanes, o_addr = s_addr + 2 * HB;
    const float scale2 = p.scale * LD_LOG2E;
    const int key = warp * 16 + lane;  // of the chunk: lanes 0..15
    float ref[HB], sum[HB];  // of all keys: the reference; of this thread's keys: the sum of weights
    // the sink is a key without a value: its weight starts the denominator (of one split, in one thread)
    const bool sunk = p.sink != nullptr && split == 0;
#pragma unroll
    for (int g = 0; g < HB; ++g) {
      ref[g] = sunk && g < nh ? p.sink[h0 + g] * LD_LOG2E : -INFINITY;
      sum[g] = sunk && g < nh && tid == 0 ? 1.f : 0.f;
    }
    bool ok = true;
    for (int c = 0; c < n_chunks; ++c) {
      // P of chunk c - 2 was read by its product
      if (*abort_flag || !mbar_wait(&s_full[c & 1], (c >> 1) & 1) || (c > 1 && !mbar_wait(&o_full[c & 1], ((c >> 1) - 1) & 1))) {
        report_error(p.status, ERR_WAIT_TMEM_FULL, c);
        *abort_flag = 1;
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);  // the lanes of a warp share its TMEM accesses
      float sc[HB];
      bool grown = false;
      if (ok) {
        tc_fence_after();
        uint32_t v[HB];
        ld_cols<HB>(s_addr + (c & 1) * HB, v);
        tmem_ld_wait();
        const int at = (c_begin + c) * LD_KEYS + key;
        const bool valid = lane < 16 && at < len && at >= key_lo;
#pragma unroll
        for (int g = 0; g < HB; ++g) {
          sc[g] = valid ? __uint_as_float(v[g]) * scale2 : -INFINITY;
          grown |= sc[g] > ref[g] + LD_SLACK;
        }
      }
      if (ld_bar_or(grown || !ok)) {  // rare after the first chunk: move the references that were outgrown
        // all 128 threads stop together
        if (c > 0 && ok && (*abort_flag || !mbar_wait(&o_full[(c - 1) & 1], ((c - 1) >> 1) & 1))) {
          report_error(p.status, ERR_WAIT_TMEM_FULL, 2000 + c);
          *abort_flag = 1;
          ok = false;
        }
        ok = !ld_bar_or(!ok);
        if (!ok) break;
        tc_fence_after();
        float alpha[HB];
#pragma unroll
        for (int g = 0; g < HB; ++g) {
          const float wm = warp_reduce_max(sc[g]);
          if (lane == 0) red_s[g][warp] = wm;
        }
        ld_bar();
#pragma unroll
        for (int g = 0; g < HB; ++g) {
          const float m = fmaxf(fmaxf(red_s[g][0], red_s[g][1]), fmaxf(red_s[g][2], red_s[g][3]));
          const bool move = m > ref[g] + LD_SLACK;
          alpha[g] = move ? exp2f(ref[g] - m) : 1.f;  // exp2(-inf) = 0: nothing seen before
          sum[g] *= alpha[g];
          ref[g] = move ? m : ref[g];
        }
        if (c > 0) {  // the previous chunk's product has completed: O is at rest
          for (int v = 0; v < 2 * v_blocks; ++v) {
            uint32_t o[HB];
            ld_cols<HB>(o_addr + v * HB, o);
            tmem_ld_wait();
#pragma unroll
            for (int g = 0; g < HB; ++g) o[g] = __float_as_uint(__uint_as_float(o[g]) * alpha[g]);
            if constexpr (HB == 32) tmem_st_32x32(o_addr + v * HB, o);
            else tmem_st_32x16(o_addr + v * HB, o);
          }
          tmem_st_wait();
        }
        tc_fence_before();
        ld_bar();  // every lane's part of O is in place before the weights are handed over; red_s is free again
        tc_fence_after();
      }
      if (lane < 16) {
        uint8_t* pbuf = p_s + (c & 1) * LdCfg<HB>::P_BYTES + (key & 7) * 2;
        const uint32_t c16 = key >> 3;
#pragma unroll
        for (int g = 0; g < HB; ++g) {
          const float w = exp2f(sc[g] - ref[g]);
          sum[g] += w;
          const __nv_bfloat16 hi = __float2bfloat16(w);
          const uint32_t off = (g >> 3) * 1024 + (g & 7) * 128 + ((c16 ^ (g & 7)) << 4);
          *reinterpret_cast<__nv_bfloat16*>(pbuf + off) = hi;
          *reinterpret_cast<__nv_bfloat16*>(pbuf + off + HB * 128) = __float2bfloat16(w - __bfloat162float(hi));
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[c & 1]);
    }
    if (ok && n_chunks > 0) {
      if (*abort_flag || !mbar_wait(&o_full[(n_chunks - 1) & 1], ((n_chunks - 1) >> 1) & 1)) {
        report_error(p.status, ERR_WAIT_TMEM_FULL, 1000);
        *abort_flag = 1;
        ok = false;
      }
      ok = !ld_bar_or(!ok);
    }
    if (ok) {
#pragma unroll
      for (int g = 0; g < HB; ++g) {
        const float ws = warp_reduce_sum(sum[g]);
        if (lane == 0) sum_s[g][warp] = ws;
      }
      ld_bar();
#pragma unroll
      for (int g = 0; g < HB; ++g) sum[g] = sum_s[g][0] + sum_s[g][1] + sum_s[g][2] + sum_s[g][3];
      if (p.num_splits > 1 && tid < nh) {
        const long long i = ((long long)t * p.H + h0 + tid) * p.num_splits + split;
        float m = -INFINITY, l = 0.f;
#pragma unroll
        for (int g = 0; g < HB; ++g)
          if (g == tid) {
            m = ref[g] * LD_LN2;
            l = sum[g];
          }
        p.ml_part[2 * i] = m;
        p.ml_part[2 * i + 1] = l;
      }
      if (n_chunks > 0) {
        tc_fence_after();
        for (int v = 0; v < v_blocks; ++v) {
          uint32_t hi[HB], lo[HB];
          ld_cols<HB>(o_addr + v * 2 * HB, hi);
          ld_cols<HB>(o_addr + v * 2 * HB + HB, lo);
          tmem_ld_wait();
          const int d = v * 128 + tid;
          if (d < p.rank) {
#pragma unroll
            for (int g = 0; g < HB; ++g) {
              if (g < nh) {
                const float o = __uint_as_float(hi[g]) + __uint_as_float(lo[g]);
                const long long row = (long long)t * p.H + h0 + g;
                if (p.num_splits == 1) p.out[row * p.rank + d] = __float2bfloat16(o / sum[g]);
                else p.o_part[(row * p.num_splits + split) * p.rank + d] = o;
              }
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
    tmem_dealloc(tmem, LdCfg<HB>::TMEM);
  }
}

}  // namespace vb

using namespace vb;

// out[t, h, n] = sum_k a[t, h, k] B_h[n, k] for n < N (B stored [H, N, K], or [H, K, N] with b_mn), times
// sigmoid(gate[t, h * N + n]) when gate is given (gate_w 1: sigmoid(gate[t, h])); then `tail` elements a[t, h, K ...], then zeros up to `width`.
// bf16; K, N, width and all strides are multiples of 8, all bases 16-byte aligned.
extern "C" int vb_head_gemm(const void* a, long long a_t, long long a_h, const void* b, int b_mn, void* out, long long o_t,
                            long long o_h, const void* gate, long long gate_stride, int gate_w, int T, int H, int K, int N,
                            int tail, int width, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (gate != nullptr && gate_w != 1 && (gate_w != N || (gate_stride & 7) || (reinterpret_cast<uintptr_t>(gate) & 15))) return -3;
  if (H <= 0 || H > 65535 || K <= 0 || N <= 0 || (K & 7) || (N & 7) || (width & 7) || width < N + tail || (a_t & 7) ||
      (a_h & 7) || (o_t & 7) || (o_h & 7) || (T + 127) / 128 > 65535 || (reinterpret_cast<uintptr_t>(out) & 15))
    return -3;
  CUtensorMap tmA, tmB;
  int rc = vb_make_tmap_3d(&tmA, a, 2, K, H, T, (uint64_t)a_h * 2, (uint64_t)a_t * 2, 64, 1, 128);
  if (rc) return rc;
  rc = b_mn ? vb_make_tmap_3d(&tmB, b, 2, N, K, H, (uint64_t)N * 2, (uint64_t)N * K * 2, 64, 64, 1)
            : vb_make_tmap_3d(&tmB, b, 2, K, N, H, (uint64_t)K * 2, (uint64_t)N * K * 2, 64, 64, 1);
  if (rc) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(head_gemm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, HG_SMEM));
    attr_set = true;
  }
  HeadGemmParams p{reinterpret_cast<const __nv_bfloat16*>(a), a_t, a_h, reinterpret_cast<__nv_bfloat16*>(out), o_t, o_h,
                   reinterpret_cast<const __nv_bfloat16*>(gate), gate_stride, gate_w, T, K, N, tail, width, b_mn, status};
  rc = (int)vb_launch_pdl(head_gemm_kernel, dim3((N + 63) / 64, H, (T + 127) / 128), dim3(HG_THREADS), HG_SMEM, stream, 1, tmA,
                          tmB, p);
  vb_count_launch();
  return rc ? rc : (int)cudaGetLastError();
}

static inline int ld_heads(int H) { return H <= 16 ? 16 : 32; }
// Stages that fit beside Q and P.
static int ld_stages(int hb, int parts) {
  int s = LD_MAX_STAGES;
  while (s > 0 && (hb == 32 ? LdCfg<32>::bytes(s, parts) : LdCfg<16>::bytes(s, parts)) > 227 * 1024) --s;
  return s;
}

extern "C" int vb_latent_decode_supported(int H, int width, int rank, int block_size) {
  return H > 0 && rank > 0 && rank <= 512 && width >= rank && (width & 63) == 0 && width / 64 <= LD_MAX_PARTS && block_size >= 8 &&
         (block_size & (block_size - 1)) == 0 && ld_stages(ld_heads(H), width / 64) >= 2;
}

// Splits of the keys that fill the SMs (one CTA each) for T rows over up to `chunks` blocks of 64 keys.
extern "C" int vb_latent_decode_splits(int T, int H, int chunks) {
  const int sms = vb_num_sms(), items = T * ((H + ld_heads(H) - 1) / ld_heads(H));
  int best = 1;
  float best_cost = 0.f;
  for (int s = 1; s <= 16 && s <= chunks; ++s) {
    const int waves = (items * s + sms - 1) / sms;
    const float cost = waves * ((chunks + s - 1) / s + 3.f) + (s > 1 ? 2.f + 0.04f * items * s / sms : 0.f);
    if (s == 1 || cost < best_cost) {
      best = s;
      best_cost = cost;
    }
  }
  return best;
}

int vb_decode_merge(const float* o_part, const float* ml_part, int B, int Hq, int D, int num_splits, void* out,
                    long long out_stride, const void* gate, long long gate_stride, int gate_w, cudaStream_t stream);

// Row t of q [T, H, width] is one of the last positions of its sequence (cu_q [B + 1], seq_lens [B]; T == B: one row each) and
// sees the page rows [num_blocks, block_size, width] up to its own (window > 0: the last `window` of them); the first `rank`
// numbers of a row are the value. sink [H] fp32 or null: exp(sink[h]) joins the denominator.
// out [T, H, rank]. work: T * H * num_splits * (rank + 2) floats (unused when num_splits == 1).
extern "C" int vb_latent_decode(const void* q, const void* pages, int num_blocks, const int* block_table, int max_blocks,
                                const int* cu_q, const int* seq_lens, int T, int B, int H, int width, int rank,
                                int block_size, float scale, int window, const float* sink, int num_splits, void* out,
                                float* work, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (!vb_latent_decode_supported(H, width, rank, block_size) || num_splits < 1 || num_splits > 65535 ||
      (num_splits > 1 && work == nullptr) || (reinterpret_cast<uintptr_t>(q) & 15))
    return -3;
  CUtensorMap tmC;
  // [64 columns] x [rows] x [parts]: one copy takes all parts of eight rows
  const int hb = ld_heads(H), parts = width / 64, stages = ld_stages(hb, parts);
  int rc = vb_make_tmap_3d(&tmC, pages, 2, 64, (uint64_t)num_blocks * block_size, parts, (uint64_t)width * 2, 128, 64, 8, parts);
  if (rc) return rc;
  LatentDecodeParams p{};
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.block_table = block_table; p.cu_q = cu_q; p.seq_lens = seq_lens; p.max_blocks = max_blocks;
  p.T = T; p.B = B; p.H = H; p.width = width; p.rank = rank; p.block_size = block_size;
  p.num_splits = num_splits; p.stages = stages; p.scale = scale; p.window = window; p.sink = sink;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.o_part = work;
  p.ml_part = work ? work + (long long)T * H * num_splits * rank : nullptr;
  p.status = status;
  static bool attr_set = false;
  if (!attr_set) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(latent_decode_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    VB_CUDA_CHECK(cudaFuncSetAttribute(latent_decode_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    attr_set = true;
  }
  const dim3 grid(T, (H + hb - 1) / hb, num_splits);
  const int smem = hb == 32 ? LdCfg<32>::bytes(stages, parts) : LdCfg<16>::bytes(stages, parts);
  rc = hb == 32 ? (int)vb_launch_pdl(latent_decode_kernel<32>, grid, dim3(LD_THREADS), (size_t)smem, stream, 1, tmC, p)
                : (int)vb_launch_pdl(latent_decode_kernel<16>, grid, dim3(LD_THREADS), (size_t)smem, stream, 1, tmC, p);
  vb_count_launch(num_splits > 1 ? 2 : 1);
  if (rc == 0) rc = (int)cudaGetLastError();
  if (rc || num_splits == 1) return rc;
  return vb_decode_merge(p.o_part, p.ml_part, T, H, rank, num_splits, out, (long long)H * rank, nullptr, 0, 0, stream);
}
