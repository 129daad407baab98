"""Gated delta rule over ragged batches with per-sequence state (``csrc/delta_rule.cu``)."""

from __future__ import annotations

import torch
import torch.nn.functional as F

from . import _lib

CHUNK_MIN = 32  # portions of at least this many tokens take the chunked tensor-core form


def delta_rule(proj: torch.Tensor, conv_w: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, norm_w: torch.Tensor,
               ring: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_lens: torch.Tensor, slots: torch.Tensor,
               max_q: int, heads: int, kv_heads: int, dim: int, vdim: int, eps: float, impl: str = "auto") -> torch.Tensor:
    """Mixer output before its last projection, [T, heads * vdim].

    ``proj`` [T, q | k | v | gate | b | a (| padding)] of ragged sequences (``cu_q`` [B + 1]); ``seq_lens`` [B] = tokens of
    each sequence up to and including these; ``slots`` [B] int32 = state slot (< 0: padding row). Updates in place
    ``state`` fp32 [slots, heads, vdim, dim] and ``ring`` [slots, taps, channels] (convolution inputs, position p in row
    p % taps). Sequences that start at position 0 ignore what their slot held. ``max_q`` == 1: one token per sequence.

    ``impl`` (portions longer than a token): "chunk" = chunks of 64 tokens on the tensor cores (bf16, head sizes in
    multiples of 8, keys up to 128), "scan" = token by token in fp32, "auto" = "chunk" for bf16 portions of 32 tokens up."""
    T, B, taps = proj.shape[0], slots.numel(), conv_w.shape[1]
    C = 2 * kv_heads * dim + heads * vdim
    out = torch.empty((T, heads * vdim), dtype=proj.dtype, device=proj.device)
    if proj.is_cuda:
        qkv = gates = unit = scratch = None
        if max_q > 1:
            can = proj.dtype == torch.bfloat16 and proj.stride(0) % 8 == 0 and bool(_lib.fn("vb_delta_chunk_supported")(dim, vdim))
            if impl == "chunk" and not can:
                raise ValueError(f"the chunked delta rule does not support dim={dim} vdim={vdim} in {proj.dtype}")
            chunk = can and (impl == "chunk" or (impl == "auto" and max_q >= CHUNK_MIN))
            new = lambda *shape: torch.empty(shape, dtype=torch.float32, device=proj.device)  # noqa: E731
            gates = new(T, 2 * heads)
            if chunk:
                qkv, unit = torch.empty((T, C), dtype=torch.bfloat16, device=proj.device), new(T, 2 * kv_heads)
                scratch = torch.empty(_lib.fn("vb_delta_chunk_bytes")(T, B, heads), dtype=torch.uint8, device=proj.device)
            else:
                qkv = new(T, C)
        rc = _lib.fn("vb_delta_rule")(proj.data_ptr(), proj.stride(0), conv_w.data_ptr(), a_log.data_ptr(), dt_bias.data_ptr(),
                                      norm_w.data_ptr(), ring.data_ptr(), state.data_ptr(), cu_q.data_ptr(),
                                      seq_lens.data_ptr(), slots.data_ptr(), _lib.ptr(qkv), _lib.ptr(unit), _lib.ptr(gates),
                                      _lib.ptr(scratch), out.data_ptr(),
                                      out.stride(0), T, B, int(max_q), heads, kv_heads, dim, vdim, taps, float(eps),
                                      int(proj.dtype == torch.float32), _lib.status_word(proj.device).data_ptr(), _lib.stream())
        _lib.check(rc, "vb_delta_rule")
        return out
    cu, lens, sl = cu_q.tolist(), seq_lens.tolist(), slots.tolist()
    for b in range(B):
        lo, hi, s = cu[b], cu[b + 1], sl[b]
        if hi == lo:
            continue
        if s < 0:
            out[lo:hi] = 0
            continue
        start = lens[b] - (hi - lo)
        x = proj[lo:hi].float()
        past = [ring[s, p % taps].float() if p >= 0 else torch.zeros(C) for p in range(start - taps + 1, start)]
        inp = torch.cat([torch.stack(past), x[:, :C]]) if past else x[:, :C]
        y = F.silu(sum(inp[j : j + hi - lo] * conv_w[:, j].float() for j in range(taps)))
        for p in range(max(start, lens[b] - taps), lens[b]):
            ring[s, p % taps] = proj[lo + p - start, :C]
        nq = kv_heads * dim
        q, k = (t.reshape(-1, kv_heads, dim) for t in (y[:, :nq], y[:, nq : 2 * nq]))
        q, k = (t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6) for t in (q, k))
        rep = heads // kv_heads
        q, k = (q * dim ** -0.5).repeat_interleave(rep, 1), k.repeat_interleave(rep, 1)
        v, gate = y[:, 2 * nq :].reshape(-1, heads, vdim), x[:, C : C + heads * vdim].reshape(-1, heads, vdim)
        beta = torch.sigmoid(x[:, C + heads * vdim : C + heads * (vdim + 1)])
        a = x[:, C + heads * (vdim + 1) : C + heads * (vdim + 2)]
        g = torch.exp(-torch.exp(a_log) * F.softplus(a + dt_bias, threshold=60.0))
        S = state[s] if start > 0 else torch.zeros_like(state[s])  # [H, V, D]
        for t in range(hi - lo):
            S = S * g[t, :, None, None]
            u = beta[t, :, None] * (v[t] - torch.einsum("hvd,hd->hv", S, k[t]))
            S = S + u[:, :, None] * k[t, :, None, :]
            o = torch.einsum("hvd,hd->hv", S, q[t])
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float() * F.silu(gate[t])
            out[lo + t] = o.reshape(-1).to(out.dtype)
        state[s] = S
    return out
