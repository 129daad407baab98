// Token-wise kernels of layer-list decoders (models/hybrid.py): 32-bit residual stream with fused add + RMSNorm (of the
// stream, or of what is added to it), scaled embedding, gated linear units, query / key norms over the projection or per head
// with rotary positions, fused with the paged KV write, the same for latent attention, CUDA-core matrix products for
// 32-bit weights (and for shapes that TMA cannot describe), and a CUDA-core paged attention that takes any head size.
//
// Every kernel is a template over the activation type (bf16 when serving, fp32 for the exact mode); arithmetic is fp32.
#include "host_utils.h"
#include "rowwise.cuh"

namespace vb {

// ---------------------------------------------------------------------------------------------------------------
// res[t] = table[ids[t]] * scale (+ pos[positions[t]], n_pos rows), fp32; y (when given): the same in the table's type.
template <typename T>
__global__ void embed_scaled_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                                    float* __restrict__ res, T* __restrict__ y, int H, float scale, const T* __restrict__ pos,
                                    const long long* __restrict__ positions, int n_pos) {
  pdl_trigger();
  pdl_wait();
  const T* src = table + ids[blockIdx.x] * (long long)H;
  const T* add = pos ? pos + max(min(positions[blockIdx.x], (long long)n_pos - 1), 0ll) * H : nullptr;
  float* dst = res + (long long)blockIdx.x * H;
  if ((H & 7) == 0) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8];
      ld8(src + v * 8, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] *= scale;
      if (add) {
        float g[8];
        ld8(add + v * 8, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += g[i];
      }
      st8(dst + v * 8, f);
      if (y) st8(y + (long long)blockIdx.x * H + v * 8, f);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float f = to_f<T>(src[i]) * scale + (add ? to_f<T>(add[i]) : 0.f);
      dst[i] = f;
      if (y) y[(long long)blockIdx.x * H + i] = from_f<T>(f);
    }
  }
}

// res[t] = table[ids[t]] / sqrt(mean of its squares + eps) * w, fp32.
template <typename T>
__global__ void embed_normed_kernel(const long long* __restrict__ ids, const T* __restrict__ table, const T* __restrict__ w,
                                    float* __restrict__ res, int H, float eps) {
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  const T* src = table + ids[blockIdx.x] * (long long)H;
  float* dst = res + (long long)blockIdx.x * H;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float f = to_f<T>(src[i]);
    ss += f * f;
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, sh) / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = to_f<T>(src[i]) * inv * to_f<T>(w[i]);
}

// ---------------------------------------------------------------------------------------------------------------
// res += delta (when given); y = res / sqrt(mean(res^2) + eps) * w, or without w the residual. The residual stays fp32 in global
// memory; the row is kept in shared memory between the two passes.
template <typename T>
__global__ void add_rmsnorm_kernel(const T* __restrict__ delta, long long delta_stride, float* __restrict__ res,
                                   const T* __restrict__ w, T* __restrict__ y, int H, float eps) {
  extern __shared__ float row[];
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  float* r = res + (long long)blockIdx.x * H;
  T* out = y + (long long)blockIdx.x * H;
  const T* d = delta ? delta + (long long)blockIdx.x * delta_stride : nullptr;
  float ss = 0.f;
  const bool vec = (H & 7) == 0 && (d == nullptr || (delta_stride & 7) == 0);
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8];
      ld8(r + v * 8, f);
      if (d) {
        float g[8];
        ld8(d + v * 8, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += g[i];
        st8(r + v * 8, f);
      }
      st8(row + v * 8, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss += f[i] * f[i];
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      float f = r[i];
      if (d) {
        f += to_f<T>(d[i]);
        r[i] = f;
      }
      row[i] = f;
      ss += f * f;
    }
  }
  norm_row_out(row, ss, w, out, H, eps, vec, sh);
}

// ---------------------------------------------------------------------------------------------------------------
// res += d / sqrt(mean(d^2) + eps) * w with d = delta, or with a gate delta * sigmoid(gate); y = res, or with fw:
// y = res / sqrt(mean(res^2) + eps) * fw * fscale.
template <typename T>
__global__ void rmsnorm_add_kernel(const T* __restrict__ delta, long long delta_stride, const T* __restrict__ gate,
                                   long long gate_stride, float* __restrict__ res, const T* __restrict__ w,
                                   const T* __restrict__ fw, float fscale, T* __restrict__ y, int H, float eps, bool vec) {
  extern __shared__ float row[];
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  const T* d = delta + (long long)blockIdx.x * delta_stride;
  const T* g = gate ? gate + (long long)blockIdx.x * gate_stride : nullptr;
  float ss = 0.f;
  if (vec) {
    for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
      float f[8];
      ld8(d + v * 8, f);
      if (g) {
        float z[8];
        ld8(g + v * 8, z);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= sigmoid_t<T>(z[i]);
      }
      st8(row + v * 8, f);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss += f[i] * f[i];
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float f = to_f<T>(d[i]) * (g ? sigmoid_t<T>(to_f<T>(g[i])) : 1.f);
      row[i] = f;
      ss += f * f;
    }
  }
  norm_row_add(row, ss, res + (long long)blockIdx.x * H, w, fw, fscale, y + (long long)blockIdx.x * H, H, eps, vec, sh);
}

// ---------------------------------------------------------------------------------------------------------------
// gu rows hold [gate (F) | up (F)]: g = min(gate, limit), u = clamp(up, -limit, limit), y = g sigmoid(alpha g) (u + 1).
template <typename T>
struct ClampedGlu {
  float limit, alpha;
  __device__ __forceinline__ float operator()(float g, float u) const {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    if (sizeof(T) == 2) return __fdividef(g, 1.f + __expf(-alpha * g)) * (u + 1.f);  // error far below a bf16 ulp
    return g / (1.f + expf(-alpha * g)) * (u + 1.f);
  }
};
// y = gelu(gate) * up with the tanh form of gelu
template <typename T>
struct GeluTanhGlu {
  __device__ __forceinline__ float operator()(float g, float u) const { return gelu_tanh<sizeof(T) == 2>(g) * u; }
};
// y = silu(gate) * up
template <typename T>
struct SiluGlu {
  __device__ __forceinline__ float operator()(float g, float u) const {
    if (sizeof(T) == 2) return __fdividef(g, 1.f + __expf(-g)) * u;
    return g / (1.f + expf(-g)) * u;
  }
};
// ROUTED: rows of a buffer sorted by expert. Gate and up of a row are multiplied with its scale first (when given); blocks of 128
// rows without an expert are left out.
template <typename T, typename Act, bool ROUTED>
__global__ void glu_kernel(const T* __restrict__ gu, long long stride, T* __restrict__ y, long long total, int F,
                           const Act act, const float* __restrict__ row_scale, const int* __restrict__ blk_expert) {
  pdl_trigger();
  pdl_wait();
  const long long step = (long long)gridDim.x * blockDim.x;
  if ((F & 7) == 0 && (stride & 7) == 0) {
    const int nv = F >> 3;
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total / 8; i += step) {
      const long long t = i / nv;
      const int c = (int)(i - t * nv) * 8;
      if (ROUTED && blk_expert[t >> 7] < 0) continue;
      const float w = ROUTED && row_scale ? row_scale[t] : 1.f;
      float g[8], u[8];
      ld8(gu + t * stride + c, g);
      ld8(gu + t * stride + F + c, u);
#pragma unroll
      for (int k = 0; k < 8; ++k) g[k] = ROUTED ? act(g[k] * w, u[k] * w) : act(g[k], u[k]);
      st8(y + t * F + c, g);
    }
  } else {
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += step) {
      const long long t = i / F;
      const int c = (int)(i - t * F);
      if (ROUTED && blk_expert[t >> 7] < 0) continue;
      const float w = ROUTED && row_scale ? row_scale[t] : 1.f;
      y[i] = from_f<T>(act(to_f<T>(gu[t * stride + c]) * w, to_f<T>(gu[t * stride + F + c]) * w));
    }
  }
}

// y[t][c] = act(x[t][c]), c < n: ACT 0: gelu with erf, 1: the square of relu. blk_expert (or null): see glu_kernel.
template <typename T, int ACT>
__global__ void activation_kernel(const T* __restrict__ x, long long stride, T* __restrict__ y, long long total, int n,
                                  const int* __restrict__ blk_expert, bool vec) {
  pdl_trigger();
  pdl_wait();
  const long long step = (long long)gridDim.x * blockDim.x, i0 = blockIdx.x * (long long)blockDim.x + threadIdx.x;
  auto act = [](float z) {
    if (ACT == 0) return gelu_erf<sizeof(T) == 2>(z);
    const float r = fmaxf(z, 0.f);
    return r * r;
  };
  const int per = vec ? n >> 3 : n;
  for (long long i = i0; i < (vec ? total / 8 : total); i += step) {
    const long long t = i / per;
    if (blk_expert && blk_expert[t >> 7] < 0) continue;
    if (vec) {
      const int c = (int)(i - t * per) * 8;
      float f[8];
      ld8(x + t * stride + c, f);
#pragma unroll
      for (int k = 0; k < 8; ++k) f[k] = act(f[k]);
      st8(y + t * n + c, f);
    } else {
      y[i] = from_f<T>(act(to_f<T>(x[t * stride + (i - t * n)])));
    }
  }
}

// y[t] = gelu(g[t]) * table[ids[t]][lo ..]. V elements per thread.
template <typename T, int V>
__global__ void gelu_rows_kernel(const T* __restrict__ g, long long g_stride, const long long* __restrict__ ids,
                                 const T* __restrict__ table, long long table_stride, int lo, T* __restrict__ y, int n,
                                 long long total) {
  pdl_trigger();
  pdl_wait();
  const int per = n / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / per;
    const int c = (int)(i - t * per) * V;
    const T *src = g + t * g_stride + c, *e = table + ids[t] * table_stride + lo + c;
    if constexpr (V == 8) {
      float a[8], b[8];
      ld8(src, a);
      ld8(e, b);
#pragma unroll
      for (int k = 0; k < 8; ++k) a[k] = gelu_tanh<sizeof(T) == 2>(a[k]) * b[k];
      st8(y + t * n + c, a);
    } else {
      y[t * n + c] = from_f<T>(gelu_tanh<sizeof(T) == 2>(to_f<T>(src[0])) * to_f<T>(e[0]));
    }
  }
}

// x = cap * tanh(x / cap)
__global__ void softcap_kernel(float* __restrict__ x, long long n, float cap) {
  pdl_trigger();
  pdl_wait();
  const long long step = (long long)gridDim.x * blockDim.x, i0 = blockIdx.x * (long long)blockDim.x + threadIdx.x;
  if ((n & 3) == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0) {
    for (long long i = i0; i < n / 4; i += step) {
      float4 v = reinterpret_cast<float4*>(x)[i];
      v = make_float4(cap * tanhf(v.x / cap), cap * tanhf(v.y / cap), cap * tanhf(v.z / cap), cap * tanhf(v.w / cap));
      reinterpret_cast<float4*>(x)[i] = v;
    }
  } else {
    for (long long i = i0; i < n; i += step) x[i] = cap * tanhf(x[i] / cap);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// One block per token. qkv row = [q (Hq * D) | k (Hk * D) | v (Hk * Dv)]. With norm weights: q and k are divided by the
// root mean square of the WHOLE projection (all heads together) and multiplied by their weights. With positions (of the
// tokens), q is multiplied by 1 + coef ln(floor((position + 1) / every) + 1). q is changed in place; k and v go to the token's place in the paged caches ([NB, Hk, BS, D] / [NB, Hk, BS, Dv]; slot < 0: no write).
template <typename T, bool VEC>
__global__ void qk_norm_kv_write_kernel(T* __restrict__ qkv, long long stride, const T* __restrict__ qw,
                                        const T* __restrict__ kw, const long long* __restrict__ slots,
                                        T* __restrict__ kc, T* __restrict__ vc, int Hq, int Hk, int D, int Dv,
                                        int block_size, float eps, const long long* __restrict__ positions, float coef,
                                        float every) {
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  T* q = qkv + (long long)blockIdx.x * stride;
  T* k = q + Hq * D;
  T* v = k + Hk * D;
  const int nq = Hq * D, nk = Hk * D, nv = Hk * Dv;
  constexpr int W = VEC ? 8 : 1;
  float iq = 1.f, ik = 1.f;
  __shared__ float temp;
  if (positions != nullptr && threadIdx.x == 0)
    temp = 1.f + coef * logf((float)floor((double)(positions[blockIdx.x] + 1) / (double)every) + 1.f);
  if (qw != nullptr) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * W; i < nq + nk; i += blockDim.x * W) {  // q and k are adjacent
      float s = 0.f;
      if (VEC) {
        float f[8];
        ld8(q + i, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) s += f[e] * f[e];
      } else {
        const float f = to_f<T>(q[i]);
        s = f * f;
      }
      if (i < nq) sq += s; else sk += s;
    }
    sq = block_sum_all(sq, sh);
    sk = block_sum_all(sk, sh);
    iq = 1.f / sqrtf(sq / (float)nq + eps);
    ik = 1.f / sqrtf(sk / (float)nk + eps);
  }
  if (positions != nullptr) {
    __syncthreads();
    iq *= temp;
  }
  if (qw != nullptr || positions != nullptr) {
    for (int i = threadIdx.x * W; i < nq; i += blockDim.x * W) {
      if (VEC) {
        float f[8], g[8];
        ld8(q + i, f);
        if (qw != nullptr) {
          ld8(qw + i, g);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] *= g[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] *= iq;
        st8(q + i, f);
      } else {
        q[i] = from_f<T>(to_f<T>(q[i]) * iq * (qw != nullptr ? to_f<T>(qw[i]) : 1.f));
      }
    }
  }
  const long long slot = slots[blockIdx.x];
  if (slot < 0) return;
  const long long blk = slot / block_size, off = slot % block_size;
  for (int i = threadIdx.x * W; i < nk; i += blockDim.x * W) {
    const int h = i / D, d = i - h * D;
    T* dst = kc + ((blk * Hk + h) * block_size + off) * (long long)D + d;
    if (VEC) {
      float f[8], g[8];
      ld8(k + i, f);
      if (kw != nullptr) {
        ld8(kw + i, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = f[e] * ik * g[e];
      }
      st8(dst, f);
    } else {
      *dst = kw != nullptr ? from_f<T>(to_f<T>(k[i]) * ik * to_f<T>(kw[i])) : k[i];
    }
  }
  for (int i = threadIdx.x * W; i < nv; i += blockDim.x * W) {
    const int h = i / Dv, d = i - h * Dv;
    T* dst = vc + ((blk * Hk + h) * block_size + off) * (long long)Dv + d;
    if (VEC) {
      float f[8];
      ld8(v + i, f);
      st8(dst, f);
    } else {
      *dst = v[i];
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Cosines and sines of position * f_i for the pairs i of a rotation, times `amp`, in shared memory. Angles are fp32.
__device__ __forceinline__ void rotation_table(float2* cs, const float* __restrict__ freqs, int n, long long pos, float amp) {
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    float sn, c;
    sincosf((float)pos * freqs[i], &sn, &c);
    cs[i] = make_float2(c * amp, sn * amp);
  }
}
constexpr int ROT_MAX = 256;  // pairs of a rotation

// One block per token. qkv row = [q (Hq * D) | k (Hk * D) | v (Hk * Dv) | ...]: every q and k head is divided by its root mean
// square and multiplied by the weight of size D that all heads share (no weights: left as it is), then its first 2 * n_rot
// dimensions turn. q in place; k and v go to the token's place in the paged caches (slot < 0: no write). v_off: where the
// values start in the row (at the keys themselves when those are the values; they are only read).
// VEC: 8 elements per lane, `lanes` lanes per head (adjacent pairs only). Otherwise a warp per head with its row in shared memory.
template <typename T, bool VEC>
__global__ void head_norm_rope_kv_write_kernel(T* __restrict__ qkv, long long stride, const T* __restrict__ qw,
                                               const T* __restrict__ kw, const float* __restrict__ freqs, int n_rot,
                                               int interleaved, float amp, const long long* __restrict__ positions,
                                               const long long* __restrict__ slots, T* __restrict__ kc, T* __restrict__ vc,
                                               int Hq, int Hk, int D, int Dv, int block_size, int v_off, float eps, int lanes) {
  __shared__ float2 cs[ROT_MAX];
  extern __shared__ float rows[];
  pdl_trigger();
  pdl_wait();
  T* base = qkv + (long long)blockIdx.x * stride;
  const long long slot = slots[blockIdx.x];
  const long long blk = slot / block_size, off = slot % block_size;
  rotation_table(cs, freqs, n_rot, positions[blockIdx.x], amp);
  __syncthreads();
  auto k_dst = [&](int hk) { return kc + ((blk * Hk + hk) * block_size + off) * (long long)D; };
  if (VEC) {
    const int per_block = blockDim.x / lanes, sub = threadIdx.x / lanes, e0 = (threadIdx.x % lanes) * 8;
    for (int h0 = 0; h0 < Hq + Hk; h0 += per_block) {  // uniform trip count: the lanes of a warp shuffle together
      const int h = h0 + sub;
      const bool on = h < Hq + Hk && e0 < D;
      float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      T* src = base + (long long)h * D + e0;  // k follows q
      if (on) ld8(src, f);
      const T* w = h < Hq ? qw : kw;
      if (qw != nullptr) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) ss += f[i] * f[i];
        for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.f / sqrtf(ss / (float)D + eps);
        if (on) {
          float g[8];
          ld8(w + e0, g);
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = f[i] * inv * g[i];
        }
      }
      if (!on) continue;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if ((e0 >> 1) + i < n_rot) {
          const float2 c = cs[(e0 >> 1) + i];
          const float u = f[2 * i], v = f[2 * i + 1];
          f[2 * i] = u * c.x - v * c.y;
          f[2 * i + 1] = v * c.x + u * c.y;
        }
      }
      if (h < Hq) st8(src, f);
      else if (slot >= 0) st8(k_dst(h - Hq) + e0, f);
    }
  } else {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* row = rows + warp * D;
    for (int h = warp; h < Hq + Hk; h += blockDim.x >> 5) {
      T* src = base + (long long)h * D;
      const T* w = h < Hq ? qw : kw;
      float ss = 0.f;
      for (int d = lane; d < D; d += 32) {
        const float f = to_f<T>(src[d]);
        row[d] = f;
        ss += f * f;
      }
      ss = warp_reduce_sum(ss);
      __syncwarp();
      const float inv = 1.f / sqrtf(ss / (float)D + eps);
      auto at = [&](int d) { return w != nullptr ? row[d] * inv * to_f<T>(w[d]) : row[d]; };
      if (h >= Hq && slot < 0) continue;
      T* dst = h < Hq ? src : k_dst(h - Hq);
      for (int d = lane; d < D; d += 32) {
        float f = at(d);
        if (d < 2 * n_rot) {
          const int i = interleaved ? d >> 1 : d % n_rot;
          const bool second = interleaved ? (d & 1) != 0 : d >= n_rot;
          const float other = at(interleaved ? d ^ 1 : (second ? d - n_rot : d + n_rot));
          f = second ? f * cs[i].x + other * cs[i].y : f * cs[i].x - other * cs[i].y;
        }
        dst[d] = from_f<T>(f);
      }
      __syncwarp();
    }
  }
  if (slot < 0) return;
  const T* v = base + v_off;
  constexpr int W = VEC ? 8 : 1;
  for (int i = threadIdx.x * W; i < Hk * Dv; i += blockDim.x * W) {
    const int h = i / Dv, d = i - h * Dv;
    T* dst = vc + ((blk * Hk + h) * block_size + off) * (long long)Dv + d;
    if (VEC) {
      float f[8];
      ld8(v + i, f);
      st8(dst, f);
    } else {
      *dst = v[i];
    }
  }
}

// Turns `rot` numbers at src into dst, the threads of the block together with `n` heads `stride` apart; pair i = (2 i, 2 i + 1) or
// (i, i + rot / 2). VEC: eight numbers at a time.
template <typename T, bool VEC>
__device__ __forceinline__ void turn_heads(const T* src, T* dst, int n, long long src_stride, long long dst_stride, int rot,
                                           bool interleaved, const float2* cs) {
  const int half = rot >> 1;
  if (interleaved) {
    constexpr int P = VEC ? 4 : 1;  // pairs at a time
    const int per = half / P;
    for (int j = threadIdx.x; j < n * per; j += blockDim.x) {
      const int h = j / per, i = (j - h * per) * P;
      const T* from = src + h * src_stride + 2 * i;
      T* to = dst + h * dst_stride + 2 * i;
      float f[2 * P];
      if constexpr (VEC) {
        ld8(from, f);
      } else {
        f[0] = to_f<T>(from[0]);
        f[1] = to_f<T>(from[1]);
      }
#pragma unroll
      for (int e = 0; e < P; ++e) {
        const float2 k = cs[i + e];
        const float u = f[2 * e], v = f[2 * e + 1];
        f[2 * e] = u * k.x - v * k.y;
        f[2 * e + 1] = v * k.x + u * k.y;
      }
      if constexpr (VEC) {
        st8(to, f);
      } else {
        to[0] = from_f<T>(f[0]);
        to[1] = from_f<T>(f[1]);
      }
    }
    return;
  }
  constexpr int W = VEC ? 8 : 1;
  for (int j = threadIdx.x; j < n * (half / W); j += blockDim.x) {
    const int h = j / (half / W), i = (j - h * (half / W)) * W;
    const T* from = src + h * src_stride;
    T* to = dst + h * dst_stride;
    float u[W], v[W], a[W], b[W];
    if constexpr (VEC) {
      ld8(from + i, u);
      ld8(from + half + i, v);
    } else {
      u[0] = to_f<T>(from[i]);
      v[0] = to_f<T>(from[half + i]);
    }
#pragma unroll
    for (int e = 0; e < W; ++e) {
      const float2 k = cs[i + e];
      a[e] = u[e] * k.x - v[e] * k.y;
      b[e] = v[e] * k.x + u[e] * k.y;
    }
    if constexpr (VEC) {
      st8(to + i, a);
      st8(to + half + i, b);
    } else {
      to[i] = from_f<T>(a[0]);
      to[half + i] = from_f<T>(b[0]);
    }
  }
}

// dst = src / sqrt(mean(src^2) + eps) * w over the block (dst may be src).
template <typename T, bool VEC>
__device__ __forceinline__ void norm_to(const T* src, T* dst, const T* __restrict__ w, int n, float eps, float* sh) {
  constexpr int W = VEC ? 8 : 1;
  float ss = 0.f;
  for (int i = threadIdx.x * W; i < n; i += blockDim.x * W) {
    float f[W];
    if constexpr (VEC) ld8(src + i, f); else f[0] = to_f<T>(src[i]);
#pragma unroll
    for (int e = 0; e < W; ++e) ss += f[e] * f[e];
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, sh) / (float)n + eps);
  for (int i = threadIdx.x * W; i < n; i += blockDim.x * W) {
    float f[W], g[W];
    if constexpr (VEC) {
      ld8(src + i, f);
      ld8(w + i, g);
    } else {
      f[0] = to_f<T>(src[i]);
      g[0] = to_f<T>(w[i]);
    }
#pragma unroll
    for (int e = 0; e < W; ++e) f[e] = f[e] * inv * g[e];
    if constexpr (VEC) st8(dst + i, f); else dst[i] = from_f<T>(f[0]);
  }
}

// One block per token. proj row = [q (H heads of dim + rot), or the queries' latent (q_rank) | latent (rank) | rotated key (rot)
// | ...]: the rotated parts turn, q in place; normed latent and rotated key go to the token's row of the pages; the queries'
// latent is normed in place.
template <typename T, bool VEC>
__global__ void latent_rope_write_kernel(T* __restrict__ proj, long long stride, const T* __restrict__ w,
                                         const float* __restrict__ freqs, float amp, int interleaved,
                                         const long long* __restrict__ positions, const long long* __restrict__ slots,
                                         T* __restrict__ pages, int width, int H, int dim, int rot, int rank, int q_rank,
                                         const T* __restrict__ qw, float eps) {
  __shared__ float2 cs[ROT_MAX];
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  T* base = proj + (long long)blockIdx.x * stride;
  const T* c = base + (q_rank ? q_rank : H * (dim + rot));
  const long long slot = slots[blockIdx.x];
  rotation_table(cs, freqs, rot >> 1, positions[blockIdx.x], amp);
  __syncthreads();
  T* dst = pages + slot * width;
  turn_heads<T, VEC>(base + dim, base + dim, H, dim + rot, dim + rot, rot, interleaved, cs);
  if (slot >= 0) turn_heads<T, VEC>(c + rank, dst + rank, 1, 0, 0, rot, interleaved, cs);
  if (q_rank) norm_to<T, VEC>(base, base, qw, q_rank, eps, sh);
  if (slot >= 0) norm_to<T, VEC>(c, dst, w, rank, eps, sh);  // uniform for the block
}

// The rotated parts of q rows [H heads of dim + rot | ...] turn in place. One block per token.
template <typename T, bool VEC>
__global__ void rotate_tails_kernel(T* __restrict__ q, long long stride, const float* __restrict__ freqs, float amp,
                                    int interleaved, const long long* __restrict__ positions, int H, int dim, int rot) {
  __shared__ float2 cs[ROT_MAX];
  pdl_trigger();
  pdl_wait();
  rotation_table(cs, freqs, rot >> 1, positions[blockIdx.x], amp);
  __syncthreads();
  T* base = q + (long long)blockIdx.x * stride + dim;
  turn_heads<T, VEC>(base, base, H, dim + rot, dim + rot, rot, interleaved, cs);
}

// rows[ctx_cu[b] + i] = page row of token i of sequence b, counted from the first of its last ctx_cu[b + 1] - ctx_cu[b] tokens
// (of seq_lens[b]; null: from its first token), in 16-byte units. One warp per row.
__global__ void latent_gather_kernel(const uint4* __restrict__ pages, const int* __restrict__ block_table, int max_blocks,
                                     const int* __restrict__ ctx_cu, const int* __restrict__ seq_lens, uint4* __restrict__ rows,
                                     int total, int B, int units, int block_size) {
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= total) return;
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (ctx_cu[mid] <= r) lo = mid; else hi = mid - 1;
  }
  const int i = r - ctx_cu[lo] + (seq_lens ? seq_lens[lo] - (ctx_cu[lo + 1] - ctx_cu[lo]) : 0);
  const long long row = (long long)block_table[(long long)lo * max_blocks + i / block_size] * block_size + i % block_size;
  for (int u = lane; u < units; u += 32) rows[(long long)r * units + u] = pages[row * units + u];
}

// out[t, h, n] = sum_k a[t, h, k] b_h[k, n] for n < N (b_h stored [N, K], or [K, N] with b_mn), times sigmoid(gate[t, h * N + n])
// (gate_w 1: sigmoid(gate[t, h]));
// then `tail` elements copied from a[t, h, K ...], then zeros up to `width`. fp32 sums, one thread per element.
template <typename T>
__global__ void head_gemm_simt_kernel(const T* __restrict__ a, long long a_t, long long a_h, const T* __restrict__ b, int b_mn,
                                      T* __restrict__ out, long long o_t, long long o_h, const T* __restrict__ gate,
                                      long long gate_stride, int gate_w, int K, int N, int tail, int width) {
  pdl_trigger();
  pdl_wait();
  const int n = blockIdx.z * blockDim.x + threadIdx.x, h = blockIdx.y;
  const long long t = blockIdx.x;
  if (n >= width) return;
  const T* ar = a + t * a_t + h * a_h;
  float x = 0.f;
  if (n < N) {
    const T* br = b + (long long)h * N * K + (b_mn ? n : (long long)n * K);
    const int step = b_mn ? N : 1;
    for (int k = 0; k < K; ++k) x = fmaf(to_f<T>(ar[k]), to_f<T>(br[(long long)k * step]), x);
    if (gate) x /= 1.f + expf(-to_f<T>(gate[t * gate_stride + (gate_w == 1 ? h : (long long)h * N + n)]));
  } else if (n < N + tail) {
    x = to_f<T>(ar[K + n - N]);
  }
  out[t * o_t + h * o_h + n] = from_f<T>(x);
}

// ---------------------------------------------------------------------------------------------------------------
// C[M, N] = A[M, K] . B[N, K]^T (+ bias), fp32 accumulation on the CUDA cores. 64 x 64 tile, 4 x 4 per thread. blk_expert (or
// null): B = [experts, N, K], the rows of A belong to experts in blocks of 128 (< 0: skipped).
template <typename TA, typename TC>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const TA* __restrict__ A, const TA* __restrict__ B,
                                                        TC* __restrict__ C, const TA* __restrict__ bias, int M, int N,
                                                        int K, long long lda, long long ldb, long long ldc,
                                                        const int* __restrict__ blk_expert) {
  __shared__ float As[16][68], Bs[16][68];
  pdl_trigger();
  pdl_wait();
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  if (blk_expert) {
    const int e = blk_expert[m0 >> 7];
    if (e < 0) return;
    B += (long long)e * N * ldb;
  }
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256, r = e >> 4, c = e & 15;
      const bool ck = k0 + c < K;
      As[c][r] = (ck && m0 + r < M) ? to_f<TA>(A[(long long)(m0 + r) * lda + k0 + c]) : 0.f;
      Bs[c][r] = (ck && n0 + r < N) ? to_f<TA>(B[(long long)(n0 + r) * ldb + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 16; ++c) {
      const float4 a = *reinterpret_cast<const float4*>(&As[c][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Bs[c][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N)
        C[(long long)m * ldc + n] = from_f<TC>(acc[i][j] + (bias ? to_f<TA>(bias[n]) : 0.f));
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Paged attention over ragged queries on the CUDA cores: one warp per (token, query head), lanes across 32 keys for the
// scores and across the value dims for the weighted sum. A query at position i sees key j <= i when window <= 0, or
// i - j < window, or j < keep_first (chunk > 0: when i / chunk == j / chunk); bias[h][min(i - j, bias_len - 1)] is added to
// the scaled score, softcap > 0 bounds it, exp(sink[h]) joins the denominator, sigmoid(gate) multiplies the result. With shift
// there is no softmax: a key weighs sigmoid(score - r1[h] ln(1 + r2[h] (i - j)) + shift[h]).
struct PagedSimtParams {
  const int* cu_q;
  const int* seq_lens;
  const int* block_table;
  long long q_stride, out_stride, gate_stride;
  int max_blocks, B, Hq, Hk, D, Dv, v_width, block_size, window, keep_first, chunk, bias_len;  // v_width: elements of a value row
  float scale, softcap;
  const float *bias, *sink;
  const float *shift, *r1, *r2;  // [Hq] or null
  const void* gate;  // [T, Hq * Dv] (gate_w 1: [T, Hq]) of the activation type, or null
  int gate_w;
};
constexpr int PS_WARPS = 4, PS_MAX_D = 1024;

template <typename T, int PS_VREG>
__global__ void __launch_bounds__(PS_WARPS * 32)
paged_attn_simt_kernel(const T* __restrict__ q, const T* __restrict__ kc, const T* __restrict__ vc, T* __restrict__ out,
                       const PagedSimtParams p) {
  __shared__ float q_s[PS_WARPS][PS_MAX_D];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * PS_WARPS + warp, t = blockIdx.x;
  if (h >= p.Hq) return;
  int lo = 0, hi = p.B - 1;  // sequence of token t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int b = lo;
  const int pos = p.seq_lens[b] - (p.cu_q[b + 1] - t);
  const int hk = h / (p.Hq / p.Hk);
  const T* qr = q + (long long)t * p.q_stride + (long long)h * p.D;
  for (int d = lane; d < p.D; d += 32) q_s[warp][d] = to_f<T>(qr[d]);
  __syncwarp();
  const int* bt = p.block_table + (long long)b * p.max_blocks;
  const float* bias = p.bias ? p.bias + (long long)h * p.bias_len : nullptr;
  const bool sig = p.shift != nullptr;
  const float shift = sig ? p.shift[h] : 0.f, r1 = p.r1 ? p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f;
  float m = sig ? 0.f : p.sink ? p.sink[h] : -INFINITY, l = sig || p.sink ? 1.f : 0.f, acc[PS_VREG];
#pragma unroll
  for (int i = 0; i < PS_VREG; ++i) acc[i] = 0.f;
  const int n = pos + 1;
  // first key of the window or chunk
  const int w_lo = p.window > 0 ? max(0, n - p.window) : p.chunk > 0 ? pos - pos % p.chunk : 0;
  const int keep = min(p.window > 0 ? p.keep_first : 0, w_lo);   // kept keys in front of it
  const int total = keep + n - w_lo;
  for (int c = 0; c < total; c += 32) {
    const int idx = c + lane;
    const bool valid = idx < total;
    const int key = idx < keep ? idx : w_lo + idx - keep;
    long long row = 0;
    float s = -INFINITY;
    if (valid) {
      row = ((long long)bt[key / p.block_size] * p.Hk + hk) * p.block_size + key % p.block_size;
      const T* kr = kc + row * p.D;
      float a = 0.f;
      for (int d = 0; d < p.D; ++d) a = fmaf(q_s[warp][d], to_f<T>(kr[d]), a);
      s = a * p.scale;
      if (bias) s += bias[min(pos - key, p.bias_len - 1)];
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      if (sig) s += shift - (p.r1 ? r1 * log1pf(r2 * (float)(pos - key)) : 0.f);
    }
    float w;
    if (sig) {
      w = valid ? sigmoid_f(s) : 0.f;
    } else {
      const float nm = fmaxf(m, warp_reduce_max(s));
      const float alpha = expf(m - nm);
      w = valid ? expf(s - nm) : 0.f;
      l = l * alpha + warp_reduce_sum(w);
      m = nm;
#pragma unroll
      for (int i = 0; i < PS_VREG; ++i) acc[i] *= alpha;
    }
    const int cnt = min(32, total - c);
    for (int j = 0; j < cnt; ++j) {
      const float wj = __shfl_sync(0xffffffffu, w, j);
      const T* vr = vc + __shfl_sync(0xffffffffu, row, j) * p.v_width;
#pragma unroll
      for (int i = 0; i < PS_VREG; ++i)
        if (lane + 32 * i < p.Dv) acc[i] = fmaf(wj, to_f<T>(vr[lane + 32 * i]), acc[i]);
    }
  }
  T* o = out + (long long)t * p.out_stride + (long long)h * p.Dv;
#pragma unroll
  for (int i = 0; i < PS_VREG; ++i) {
    const int d = lane + 32 * i;
    if (d >= p.Dv) continue;
    float x = acc[i] / l;
    if (p.gate)
      x /= 1.f + expf(-to_f<T>(reinterpret_cast<const T*>(p.gate)[t * p.gate_stride + (p.gate_w == 1 ? h : (long long)h * p.Dv + d)]));
    o[d] = from_f<T>(x);
  }
}

}  // namespace vb

using namespace vb;
typedef __nv_bfloat16 bf16;

// pos (n_pos rows, with the tokens' positions) or null
extern "C" int vb_embed_scaled(const long long* ids, const void* table, float* res, void* y, int T, int H, float scale,
                               const void* pos, const long long* positions, int n_pos, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (pos != nullptr && (positions == nullptr || n_pos <= 0)) return -3;
  const dim3 g(T), b(row_threads(H));
  if (f32) VB_DONE(vb_launch_pdl(embed_scaled_kernel<float>, g, b, 0, stream, 1, ids, (const float*)table, res, (float*)y, H,
                                scale, (const float*)pos, positions, n_pos));
  VB_DONE(vb_launch_pdl(embed_scaled_kernel<bf16>, g, b, 0, stream, 1, ids, (const bf16*)table, res, (bf16*)y, H, scale,
                        (const bf16*)pos, positions, n_pos));
}

extern "C" int vb_add_rmsnorm(const void* delta, long long delta_stride, float* res, const void* w, void* y, int T, int H,
                              float eps, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  const size_t smem = (size_t)H * 4;
  if (smem > 160 * 1024) return -3;
  const dim3 g(T), b(row_threads(H));
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(add_rmsnorm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    VB_CUDA_CHECK(cudaFuncSetAttribute(add_rmsnorm_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    attr = true;
  }
  if (f32)
    VB_DONE(vb_launch_pdl(add_rmsnorm_kernel<float>, g, b, smem, stream, 1, (const float*)delta, delta_stride, res,
                          (const float*)w, (float*)y, H, eps));
  VB_DONE(vb_launch_pdl(add_rmsnorm_kernel<bf16>, g, b, smem, stream, 1, (const bf16*)delta, delta_stride, res,
                        (const bf16*)w, (bf16*)y, H, eps));
}

template <typename T, bool ROUTED = false, typename Act>
static int launch_glu(const void* gu, long long stride, void* y, int T_, int F, const Act& act, cudaStream_t stream,
                      const float* row_scale = nullptr, const int* blk_expert = nullptr) {
  if (T_ <= 0 || F <= 0) return 0;
  const long long total = (long long)T_ * F;
  long long blocks = (total / 8 + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (blocks < 1) blocks = 1;
  VB_DONE(vb_launch_pdl(glu_kernel<T, Act, ROUTED>, dim3((unsigned)blocks), dim3(256), 0, stream, 1, (const T*)gu, stride,
                        (T*)y, total, F, act, row_scale, blk_expert));
}

// blk_expert (T / 128 of them) or null: rows of a buffer sorted by expert; row_scale [T] or null: see glu_kernel.
extern "C" int vb_silu_glu(const void* gu, long long stride, void* y, int T, int F, const float* row_scale,
                           const int* blk_expert, int f32, cudaStream_t stream) {
  if (blk_expert) {
    if (f32) return launch_glu<float, true>(gu, stride, y, T, F, SiluGlu<float>{}, stream, row_scale, blk_expert);
    return launch_glu<bf16, true>(gu, stride, y, T, F, SiluGlu<bf16>{}, stream, row_scale, blk_expert);
  }
  if (row_scale) return -3;
  if (f32) return launch_glu<float>(gu, stride, y, T, F, SiluGlu<float>{}, stream);
  return launch_glu<bf16>(gu, stride, y, T, F, SiluGlu<bf16>{}, stream);
}

// y [T, n] = act of the first n elements of a row: 0 gelu with erf, 1 the square of relu. blk_expert (T / 128 of them) or null.
extern "C" int vb_activation(const void* x, long long stride, void* y, int T, int n, int act, const int* blk_expert, int f32,
                             cudaStream_t stream) {
  if (T <= 0 || n <= 0) return 0;
  if (act < 0 || act > 1) return -3;
  const long long total = (long long)T * n;
  const bool vec = ((n | stride) & 7) == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0;
  const dim3 grid((unsigned)max(1ll, min((total / 8 + 255) / 256, 148ll * 16))), b(256);
#define VB_ACT(TT, A) \
  VB_DONE(vb_launch_pdl(activation_kernel<TT, A>, grid, b, 0, stream, 1, (const TT*)x, stride, (TT*)y, total, n, blk_expert, vec))
  if (f32) {
    if (act == 0) VB_ACT(float, 0);
    VB_ACT(float, 1);
  }
  if (act == 0) VB_ACT(bf16, 0);
  VB_ACT(bf16, 1);
#undef VB_ACT
}

// y [T, n] = gelu(g) * table[ids, lo .. lo + n)
extern "C" int vb_gelu_rows(const void* g, long long g_stride, const long long* ids, const void* table, long long table_stride,
                            int lo, void* y, int T, int n, int f32, cudaStream_t stream) {
  if (T <= 0 || n <= 0) return 0;
  const bool vec = ((n | lo | g_stride | table_stride) & 7) == 0 &&
                   ((reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(table)) & 15) == 0;
  const long long total = (long long)T * n / (vec ? 8 : 1);
  const dim3 grid((unsigned)min((total + 127) / 128, 148ll * 16)), b(128);
#define VB_GR(TT, V)                                                                                                  \
  VB_DONE(vb_launch_pdl(gelu_rows_kernel<TT, V>, grid, b, 0, stream, 1, (const TT*)g, g_stride, ids, (const TT*)table, \
                        table_stride, lo, (TT*)y, n, total))
  if (f32) {
    if (vec) VB_GR(float, 8);
    VB_GR(float, 1);
  }
  if (vec) VB_GR(bf16, 8);
  VB_GR(bf16, 1);
#undef VB_GR
}

extern "C" int vb_softcap(float* x, long long n, float cap, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (!(cap > 0.f)) return -3;
  long long blocks = (n + 1023) / 1024;
  if (blocks > 148 * 16) blocks = 148 * 16;
  VB_DONE(vb_launch_pdl(softcap_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, 1, x, n, cap));
}

extern "C" int vb_embed_normed(const long long* ids, const void* table, const void* w, float* res, int T, int H, float eps,
                               int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  const dim3 g(T), b(row_threads(H));
  if (f32)
    VB_DONE(vb_launch_pdl(embed_normed_kernel<float>, g, b, 0, stream, 1, ids, (const float*)table, (const float*)w, res, H, eps));
  VB_DONE(vb_launch_pdl(embed_normed_kernel<bf16>, g, b, 0, stream, 1, ids, (const bf16*)table, (const bf16*)w, res, H, eps));
}

extern "C" int vb_clamped_glu(const void* gu, long long stride, void* y, int T, int F, float limit, float alpha, int f32,
                              cudaStream_t stream) {
  if (f32) return launch_glu<float>(gu, stride, y, T, F, ClampedGlu<float>{limit, alpha}, stream);
  return launch_glu<bf16>(gu, stride, y, T, F, ClampedGlu<bf16>{limit, alpha}, stream);
}

extern "C" int vb_gelu_glu(const void* gu, long long stride, void* y, int T, int F, int f32, cudaStream_t stream) {
  if (f32) return launch_glu<float>(gu, stride, y, T, F, GeluTanhGlu<float>{}, stream);
  return launch_glu<bf16>(gu, stride, y, T, F, GeluTanhGlu<bf16>{}, stream);
}

// delta rows of delta_stride elements, gate rows (or null) of gate_stride; fw null: y = the new residual in the activation type.
extern "C" int vb_rmsnorm_add(const void* delta, long long delta_stride, const void* gate, long long gate_stride, float* res,
                              const void* w, const void* fw, float fscale, void* y, int T, int H, float eps, int f32,
                              cudaStream_t stream) {
  if (T <= 0) return 0;
  const size_t smem = (size_t)H * 4;
  if (smem > 160 * 1024) return -3;
  const bool vec = ((H | delta_stride | gate_stride) & 7) == 0 &&
                   ((reinterpret_cast<uintptr_t>(delta) | reinterpret_cast<uintptr_t>(gate)) & 15) == 0;
  const dim3 g(T), b(row_threads(H));
  static bool attr = false;
  if (!attr) {
    VB_CUDA_CHECK(cudaFuncSetAttribute(rmsnorm_add_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    VB_CUDA_CHECK(cudaFuncSetAttribute(rmsnorm_add_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    attr = true;
  }
  if (f32)
    VB_DONE(vb_launch_pdl(rmsnorm_add_kernel<float>, g, b, smem, stream, 1, (const float*)delta, delta_stride, (const float*)gate,
                          gate_stride, res, (const float*)w, (const float*)fw, fscale, (float*)y, H, eps, vec));
  VB_DONE(vb_launch_pdl(rmsnorm_add_kernel<bf16>, g, b, smem, stream, 1, (const bf16*)delta, delta_stride, (const bf16*)gate,
                        gate_stride, res, (const bf16*)w, (const bf16*)fw, fscale, (bf16*)y, H, eps, vec));
}

// qw / kw null: no norm (k and v only written to the cache). positions null: no factor of the queries.
extern "C" int vb_qk_norm_kv_write(void* qkv, long long stride, const void* qw, const void* kw, const long long* slots,
                                   void* kc, void* vc, int T, int Hq, int Hk, int D, int Dv, int block_size, float eps,
                                   const long long* positions, float coef, float every, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((qw == nullptr) != (kw == nullptr) || !(every > 0.f)) return -3;
  const bool vec = (D & 7) == 0 && (Dv & 7) == 0 && (stride & 7) == 0;
  const dim3 g(T), b(row_threads(Hq * D));
#define VB_QKN(TT, V)                                                                                              \
  VB_DONE(vb_launch_pdl(qk_norm_kv_write_kernel<TT, V>, g, b, 0, stream, 1, (TT*)qkv, stride, (const TT*)qw,       \
                        (const TT*)kw, slots, (TT*)kc, (TT*)vc, Hq, Hk, D, Dv, block_size, eps, positions, coef, every))
  if (f32) {
    if (vec) VB_QKN(float, true);
    VB_QKN(float, false);
  }
  if (vec) VB_QKN(bf16, true);
  VB_QKN(bf16, false);
#undef VB_QKN
}

// a_f32 / out_f32: element types of (A, B, bias) and of C (fp32 inputs give fp32 outputs).
extern "C" int vb_gemm_simt(const void* A, const void* B, void* C, const void* bias, int M, int N, int K, long long lda,
                            long long ldb, long long ldc, int a_f32, int out_f32, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  if (K <= 0 || (M + 63) / 64 > 65535 || (a_f32 && !out_f32)) return -3;
  const dim3 g((N + 63) / 64, (M + 63) / 64), b(256);
  if (a_f32)
    VB_DONE(vb_launch_pdl(gemm_simt_kernel<float, float>, g, b, 0, stream, 1, (const float*)A, (const float*)B, (float*)C,
                          (const float*)bias, M, N, K, lda, ldb, ldc, (const int*)nullptr));
  if (out_f32)
    VB_DONE(vb_launch_pdl(gemm_simt_kernel<bf16, float>, g, b, 0, stream, 1, (const bf16*)A, (const bf16*)B, (float*)C,
                          (const bf16*)bias, M, N, K, lda, ldb, ldc, (const int*)nullptr));
  VB_DONE(vb_launch_pdl(gemm_simt_kernel<bf16, bf16>, g, b, 0, stream, 1, (const bf16*)A, (const bf16*)B, (bf16*)C,
                        (const bf16*)bias, M, N, K, lda, ldb, ldc, (const int*)nullptr));
}

// C[rows of e] = A[rows of e] . B[e]^T, B [E, N, K]; M a multiple of 128, blk_expert [M / 128].
extern "C" int vb_grouped_gemm_simt(const void* A, const void* B, void* C, int M, int N, int K, const int* blk_expert, int f32,
                                    cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  if (K <= 0 || (M & 127) || M / 64 > 65535 || blk_expert == nullptr) return -3;
  const dim3 g((N + 63) / 64, M / 64), b(256);
  if (f32)
    VB_DONE(vb_launch_pdl(gemm_simt_kernel<float, float>, g, b, 0, stream, 1, (const float*)A, (const float*)B, (float*)C,
                          (const float*)nullptr, M, N, K, (long long)K, (long long)K, (long long)N, blk_expert));
  VB_DONE(vb_launch_pdl(gemm_simt_kernel<bf16, bf16>, g, b, 0, stream, 1, (const bf16*)A, (const bf16*)B, (bf16*)C,
                        (const bf16*)nullptr, M, N, K, (long long)K, (long long)K, (long long)N, blk_expert));
}

// Caches [NB, Hk, block_size, D] and [NB, Hk, block_size, v_width] (the first Dv elements of a row are the value).
extern "C" int vb_paged_attention_simt(const void* q, long long q_stride, const void* kc, const void* vc,
                                       const int* block_table, int max_blocks, const int* cu_q, const int* seq_lens,
                                       int T, int B, int Hq, int Hk, int D, int Dv, int v_width, int block_size, float scale,
                                       int window, int keep_first, int chunk, const float* bias, int bias_len,
                                       float softcap, const float* sink, const float* shift, const float* r1,
                                       const float* r2, const void* gate, long long gate_stride, int gate_w, void* out,
                                       long long out_stride, int f32, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if ((shift && (bias || sink || softcap > 0.f)) || (r1 && (!shift || !r2))) return -3;
  if (Hk <= 0 || Hq % Hk != 0 || D <= 0 || D > PS_MAX_D || Dv <= 0 || Dv > PS_MAX_D || v_width < Dv || (bias && bias_len <= 0))
    return -3;
  PagedSimtParams p{};
  p.cu_q = cu_q; p.seq_lens = seq_lens; p.block_table = block_table;
  p.q_stride = q_stride; p.out_stride = out_stride; p.gate_stride = gate_stride;
  p.max_blocks = max_blocks; p.B = B; p.Hq = Hq; p.Hk = Hk; p.D = D; p.Dv = Dv; p.v_width = v_width; p.block_size = block_size;
  p.window = window; p.keep_first = keep_first; p.chunk = chunk; p.bias_len = bias_len;
  p.scale = scale; p.softcap = softcap; p.bias = bias; p.sink = sink; p.gate = gate;
  p.shift = shift; p.r1 = r1; p.r2 = r2; p.gate_w = gate_w;
  const dim3 g(T, (Hq + PS_WARPS - 1) / PS_WARPS), b(PS_WARPS * 32);
#define VB_PSA(TT, V)                                                                                             \
  VB_DONE(vb_launch_pdl(paged_attn_simt_kernel<TT, V>, g, b, 0, stream, 1, (const TT*)q, (const TT*)kc, (const TT*)vc, \
                        (TT*)out, p))
  if (f32) {
    if (Dv <= 128) VB_PSA(float, 4);
    VB_PSA(float, PS_MAX_D / 32);
  }
  if (Dv <= 128) VB_PSA(bf16, 4);
  VB_PSA(bf16, PS_MAX_D / 32);
#undef VB_PSA
}

// qw / kw null: no norm. freqs: n_rot fp32 angular frequencies (n_rot 0: no rotation). key_values: no v in the row, the values
// are the keys before norm and rotation.
extern "C" int vb_head_norm_rope_kv_write(void* qkv, long long stride, const void* qw, const void* kw, const float* freqs,
                                          int n_rot, int interleaved, float amp, const long long* positions,
                                          const long long* slots, void* kc, void* vc, int T, int Hq, int Hk, int D, int Dv,
                                          int block_size, int key_values, float eps, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (key_values && D != Dv) return -3;
  const int v_off = (key_values ? Hq : Hq + Hk) * D;
  if ((qw == nullptr) != (kw == nullptr) || n_rot < 0 || n_rot > ROT_MAX || 2 * n_rot > D || D > PS_MAX_D) return -3;
  const bool vec = (D & 7) == 0 && D <= 256 && (Dv & 7) == 0 && (stride & 7) == 0 && (interleaved || n_rot == 0) &&
                   (reinterpret_cast<uintptr_t>(qkv) & 15) == 0;
  int lanes = 1;
  while (lanes * 8 < D) lanes *= 2;
  const dim3 g(T), b(vec ? 256 : 128);
  const size_t smem = vec ? 0 : 4 * (size_t)D * sizeof(float);
#define VB_HNR(TT, V)                                                                                                  \
  VB_DONE(vb_launch_pdl(head_norm_rope_kv_write_kernel<TT, V>, g, b, smem, stream, 1, (TT*)qkv, stride, (const TT*)qw, \
                        (const TT*)kw, freqs, n_rot, interleaved, amp, positions, slots, (TT*)kc, (TT*)vc, Hq, Hk, D, Dv, \
                        block_size, v_off, eps, lanes))
  if (f32) {
    if (vec) VB_HNR(float, true);
    VB_HNR(float, false);
  }
  if (vec) VB_HNR(bf16, true);
  VB_HNR(bf16, false);
#undef VB_HNR
}

// q_rank > 0 (and H 0): the row starts with the latent of the queries, normed in place with qw.
extern "C" int vb_latent_rope_write(void* proj, long long stride, const void* w, const float* freqs, float amp, int interleaved,
                                    const long long* positions, const long long* slots, void* pages, int width, int T, int H,
                                    int dim, int rot, int rank, int q_rank, const void* qw, float eps, int f32,
                                    cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot < 0 || (rot & 1) || rot > 2 * ROT_MAX || rank <= 0 || width < rank + rot || (q_rank > 0 && (H != 0 || qw == nullptr)))
    return -3;
  const bool vec = (rot & (interleaved ? 7 : 15)) == 0 && (dim & 7) == 0 && (rank & 7) == 0 && (q_rank & 7) == 0 &&
                   (width & 7) == 0 && (stride & 7) == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
  const dim3 g(T), b(128);
#define VB_LRW(TT, V)                                                                                                  \
  VB_DONE(vb_launch_pdl(latent_rope_write_kernel<TT, V>, g, b, 0, stream, 1, (TT*)proj, stride, (const TT*)w, freqs, amp, \
                        interleaved, positions, slots, (TT*)pages, width, H, dim, rot, rank, q_rank, (const TT*)qw, eps))
  if (f32) {
    if (vec) VB_LRW(float, true);
    VB_LRW(float, false);
  }
  if (vec) VB_LRW(bf16, true);
  VB_LRW(bf16, false);
#undef VB_LRW
}

extern "C" int vb_rotate_tails(void* q, long long stride, const float* freqs, float amp, int interleaved,
                               const long long* positions, int T, int H, int dim, int rot, int f32, cudaStream_t stream) {
  if (T <= 0 || H <= 0 || rot == 0) return 0;
  if (rot < 0 || (rot & 1) || rot > 2 * ROT_MAX) return -3;
  const bool vec = (rot & (interleaved ? 7 : 15)) == 0 && (dim & 7) == 0 && (stride & 7) == 0 &&
                   (reinterpret_cast<uintptr_t>(q) & 15) == 0;
  const dim3 g(T), b(128);
#define VB_RT(TT, V) \
  VB_DONE(vb_launch_pdl(rotate_tails_kernel<TT, V>, g, b, 0, stream, 1, (TT*)q, stride, freqs, amp, interleaved, positions, H, \
                        dim, rot))
  if (f32) {
    if (vec) VB_RT(float, true);
    VB_RT(float, false);
  }
  if (vec) VB_RT(bf16, true);
  VB_RT(bf16, false);
#undef VB_RT
}

// row_bytes: bytes of a page row, a multiple of 16.
extern "C" int vb_latent_gather(const void* pages, const int* block_table, int max_blocks, const int* ctx_cu,
                                const int* seq_lens, void* rows, int total, int B, int row_bytes, int block_size,
                                cudaStream_t stream) {
  if (total <= 0 || B <= 0) return 0;
  if (row_bytes & 15) return -3;
  VB_DONE(vb_launch_pdl(latent_gather_kernel, dim3((total + 7) / 8), dim3(256), 0, stream, 1, (const uint4*)pages, block_table,
                        max_blocks, ctx_cu, seq_lens, (uint4*)rows, total, B, row_bytes / 16, block_size));
}

extern "C" int vb_head_gemm_simt(const void* a, long long a_t, long long a_h, const void* b, int b_mn, void* out, long long o_t,
                                 long long o_h, const void* gate, long long gate_stride, int gate_w, int T, int H, int K, int N,
                                 int tail, int width, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || H > 65535 || K <= 0 || width < N + tail) return -3;
  const dim3 g(T, H, (width + 127) / 128), blk(128);
  if (f32)
    VB_DONE(vb_launch_pdl(head_gemm_simt_kernel<float>, g, blk, 0, stream, 1, (const float*)a, a_t, a_h, (const float*)b, b_mn,
                          (float*)out, o_t, o_h, (const float*)gate, gate_stride, gate_w, K, N, tail, width));
  VB_DONE(vb_launch_pdl(head_gemm_simt_kernel<bf16>, g, blk, 0, stream, 1, (const bf16*)a, a_t, a_h, (const bf16*)b, b_mn,
                        (bf16*)out, o_t, o_h, (const bf16*)gate, gate_stride, gate_w, K, N, tail, width));
}
