"""Gated linear attention over ragged batches with per-sequence state (``csrc/gated_linear_attention.cu``)."""

from __future__ import annotations

import torch
import torch.nn.functional as F

from . import _lib


def gated_linear_attention(proj: torch.Tensor, decay_w: torch.Tensor, decay_b: torch.Tensor, norm_w: torch.Tensor,
                           state: torch.Tensor, cu_q: torch.Tensor, seq_lens: torch.Tensor, slots: torch.Tensor, max_q: int,
                           heads: int, dim: int, vdim: int, tau: float, eps: float, *, singles: int = 0,
                           impl: str = "auto") -> torch.Tensor:
    """Mixer output before its last projection, [T, heads * vdim].

    ``proj`` [T, q | k | v | gate | r (| ...)] of ragged sequences (``cu_q`` [B + 1]), r being the ``rank`` numbers that the decay
    comes from; ``seq_lens`` [B] = tokens of each sequence up to and including these; ``slots`` [B] int32 = state slot (< 0:
    padding row). z = ``decay_w`` [heads * dim, rank] r + ``decay_b``; row d of a head's state S decays by sigmoid(z_d) ** (1 / tau),
    then k v^T is added; o = S^T q * dim ** -0.5, RMS-normed (weight ``norm_w`` [vdim]) and multiplied with silu(gate). Decays and
    state are fp32. Updates in place ``state`` fp32 [slots, heads, vdim, dim]. Sequences that start at position 0 ignore what their slot
    held. ``max_q`` == 1: one token per sequence; otherwise the leading ``singles`` sequences have one.

    ``impl`` (sequences that bring more than a token): "chunk" = chunks of 64 tokens on the tensor cores (bf16, head sizes in
    multiples of 8, keys up to 128, values up to 256, ranks up to 64), "scan" = token by token in fp32, "auto" = "chunk" where it
    applies."""
    T, B, rank = proj.shape[0], slots.numel(), decay_w.shape[1]
    if not proj.is_cuda:
        return _gla_ref(proj, decay_w, decay_b, norm_w, state, cu_q, seq_lens, slots, heads, dim, vdim, tau, eps)
    f32, dev = proj.dtype == torch.float32, proj.device
    out = torch.empty((T, heads * vdim), dtype=proj.dtype, device=dev)
    can = (not f32 and proj.stride(0) % 8 == 0 and proj.data_ptr() % 16 == 0
           and bool(_lib.fn("vb_gla_chunk_supported")(heads, dim, vdim, rank)))
    if impl == "chunk" and not can:
        raise ValueError(f"chunked linear attention does not support dim={dim} vdim={vdim} rank={rank} in {proj.dtype}")
    chunk = can and impl != "scan"
    singles = B if max_q == 1 else singles
    decay = None if chunk or singles == B else torch.empty((T, heads * dim), dtype=torch.float32, device=dev)
    rc = _lib.fn("vb_gla")(proj.data_ptr(), proj.stride(0), decay_w.data_ptr(), decay_b.data_ptr(), norm_w.data_ptr(),
                           state.data_ptr(), cu_q.data_ptr(), seq_lens.data_ptr(), slots.data_ptr(), _lib.ptr(decay),
                           out.data_ptr(), out.stride(0), T, B, singles, int(max_q), heads, dim, vdim, rank, float(tau), float(eps),
                           int(f32), int(chunk), _lib.status_word(dev).data_ptr(), _lib.stream())
    _lib.check(rc, "vb_gla")
    return out


def _gla_ref(proj, decay_w, decay_b, norm_w, state, cu_q, seq_lens, slots, H, D, V, tau, eps):
    out = torch.zeros((proj.shape[0], H * V), dtype=proj.dtype)
    cu, lens, sl = cu_q.tolist(), seq_lens.tolist(), slots.tolist()
    for b in range(len(sl)):
        lo, hi, s = cu[b], cu[b + 1], sl[b]
        if hi == lo or s < 0:
            continue
        n = hi - lo
        q, k, v, g, r = proj[lo:hi, : 2 * H * (D + V) + decay_w.shape[1]].float().split(
            [H * D, H * D, H * V, H * V, decay_w.shape[1]], 1)
        a = torch.exp(F.logsigmoid(r @ decay_w.float().t() + decay_b) / tau).view(n, H, D)
        q, k, v = q.reshape(n, H, D) * D ** -0.5, k.reshape(n, H, D), v.reshape(n, H, V)
        S = state[s] if lens[b] > n else torch.zeros_like(state[s])  # [H, V, D]
        o = torch.empty(n, H, V)
        for t in range(n):
            S = S * a[t, :, None, :] + v[t, :, :, None] * k[t, :, None, :]
            o[t] = torch.einsum("hvd,hd->hv", S, q[t])
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
        out[lo:hi] = (o.reshape(n, -1) * F.silu(g)).to(out.dtype)
        state[s] = S
    return out
