"""Latent attention over pages of latents (``csrc/latent_attention.cu``, ``csrc/flash_attention_paged.cu``).

A page row holds one token: the normed latent (``rank`` numbers), the rotated key part all heads share, zeros up to a
multiple of 64. Two forms of the same attention: short portions stay in the latent space (the up projection of the keys
is applied to the queries, that of the values to the weighted sum), longer ones expand the keys and values of their context.
"""

from __future__ import annotations

import torch

from . import _lib
from .attention import rotate_pairs


def latent_width(size: int) -> int:
    """Numbers of a page row for ``size`` of latent and rotated part."""
    return (size + 63) // 64 * 64


def latent_prefill_supported(heads: int, dim: int, rot_dim: int, vdim: int, rank: int, dtype, device) -> bool:
    """Whether :func:`latent_prefill` takes these sizes (else every portion runs in the latent space)."""
    if torch.device(device).type != "cuda":
        return True
    return dtype == torch.bfloat16 and bool(_lib.fn("vb_latent_flash_supported")(heads, dim, rot_dim, vdim, rank))


def latent_rope_write(proj: torch.Tensor, norm_w: torch.Tensor, freqs: torch.Tensor, positions: torch.Tensor,
                      slots: torch.Tensor, pages: torch.Tensor, heads: int, dim: int, rot_dim: int, rank: int, eps: float, *,
                      amplitude: float = 1.0, interleaved: bool = False, q_rank: int = 0,
                      q_norm_w: torch.Tensor | None = None) -> None:
    """``proj`` [T, q (heads x [dim | rot_dim]) | latent (rank) | rotated key (rot_dim) | ...]: rotary positions on the rotated
    parts, RMS norm of the latent, latent and rotated key to the token's place in ``pages``
    [NB, BS, latent_width(rank + rot_dim)] (slot < 0: no write). The query part of ``proj`` is changed in place. With
    ``q_rank`` (and ``heads`` 0) that part is the latent of the queries: its RMS norm times ``q_norm_w``."""
    T, nq = proj.shape[0], q_rank or heads * (dim + rot_dim)
    if q_rank and heads:
        raise ValueError("either queries or their latent")
    if proj.is_cuda:
        rc = _lib.fn("vb_latent_rope_write")(proj.data_ptr(), proj.stride(0), norm_w.data_ptr(), freqs.data_ptr(),
                                             float(amplitude), int(interleaved), positions.data_ptr(), slots.data_ptr(),
                                             pages.data_ptr(), pages.shape[2], T, heads, dim, rot_dim, rank, q_rank,
                                             _lib.ptr(q_norm_w), float(eps), int(proj.dtype == torch.float32), _lib.stream())
        _lib.check(rc, "vb_latent_rope_write")
        return
    from .nn import _rmsnorm_ref

    if q_rank:
        proj[:, :nq] = _rmsnorm_ref(proj[:, :nq].float(), q_norm_w.float(), eps).to(proj.dtype)
    else:
        rotate_tails(proj, freqs, positions, heads, dim, rot_dim, amplitude=amplitude, interleaved=interleaved)
    c = _rmsnorm_ref(proj[:, nq : nq + rank].float(), norm_w.float(), eps)
    k = rotate_pairs(proj[:, nq + rank : nq + rank + rot_dim], positions, freqs, interleaved, amplitude)
    ok = slots >= 0
    rows = torch.cat((c, k), -1).to(pages.dtype)
    pages.view(-1, pages.shape[2])[slots[ok], : rank + rot_dim] = rows[ok]


def rotate_tails(q: torch.Tensor, freqs: torch.Tensor, positions: torch.Tensor, heads: int, dim: int, rot_dim: int, *,
                 amplitude: float = 1.0, interleaved: bool = False) -> None:
    """Rotary positions on the last ``rot_dim`` dimensions of every head of ``q`` [T, heads x [dim | rot_dim] | ...], in place."""
    if q.is_cuda:
        rc = _lib.fn("vb_rotate_tails")(q.data_ptr(), q.stride(0), freqs.data_ptr(), float(amplitude), int(interleaved),
                                        positions.data_ptr(), q.shape[0], heads, dim, rot_dim, int(q.dtype == torch.float32),
                                        _lib.stream())
        _lib.check(rc, "vb_rotate_tails")
        return
    t = q[:, : heads * (dim + rot_dim)].view(q.shape[0], heads, dim + rot_dim)[..., dim:]
    t.copy_(rotate_pairs(t, positions, freqs, interleaved, amplitude))


def _times_gate(o: torch.Tensor, gate: torch.Tensor | None, heads: int) -> torch.Tensor:
    """o [T, heads * n] times the sigmoid of ``gate`` [T, heads * n] or [T, heads]."""
    if gate is None:
        return o
    g = torch.sigmoid(gate.float())
    return o * (g if g.shape[1] == o.shape[1] else g.repeat_interleave(o.shape[1] // heads, 1))


def latent_queries(q: torch.Tensor, uk: torch.Tensor, impl: str = "auto") -> torch.Tensor:
    """q [T, H, dim + rot_dim], uk [H, dim, rank] -> [T, H, latent_width(rank + rot_dim)]: queries against latents, rotated part."""
    T, H, D = q.shape
    dim, rank = uk.shape[1:]
    rot = D - dim
    width = latent_width(rank + rot)
    if q.is_cuda:
        out = torch.empty((T, H, width), dtype=q.dtype, device=q.device)
        _head_gemm(q, uk, out, True, dim, rank, rot, None, impl)
        return out
    out = q.new_zeros((T, H, width))
    out[..., :rank] = torch.einsum("thd,hdr->thr", q[..., :dim].float(), uk.float())
    out[..., rank : rank + rot] = q[..., dim:]
    return out


def latent_values(lat: torch.Tensor, uv: torch.Tensor, gate: torch.Tensor | None, out: torch.Tensor,
                  impl: str = "auto") -> torch.Tensor:
    """lat [T, H, rank], uv [H, vdim, rank] -> ``out`` [T, H * vdim], times the sigmoid of ``gate`` [T, H * vdim] (or [T, H]: one
    number per head)."""
    T, H, rank = lat.shape
    vdim = uv.shape[1]
    if lat.is_cuda:
        _head_gemm(lat, uv, out.view(T, H, vdim), False, rank, vdim, 0, gate, impl)
        return out
    o = torch.einsum("thr,hvr->thv", lat.float(), uv.float()).reshape(T, -1)
    out.copy_(_times_gate(o, gate, H))
    return out


def _gate_width(gate, heads: int, size: int) -> int:
    """Numbers of ``gate`` per head: one, or one for each of the head's ``size`` outputs."""
    if gate is not None and gate.shape[1] not in (heads, heads * size):
        raise ValueError(f"a gate of {gate.shape[1]} for {heads} heads of {size}")
    return 1 if gate is not None and gate.shape[1] == heads else size


def _head_gemm(a, b, out, b_mn: bool, K: int, N: int, tail: int, gate, impl: str) -> None:
    """out[t, h, :N] = a[t, h, :K] . B_h (b [H, N, K], or [H, K, N] with ``b_mn``); out[t, h, N:] = a[t, h, K : K + tail],
    zeros behind it."""
    T, H, _ = a.shape
    if a.stride(2) != 1 or out.stride(2) != 1 or a.stride(1) != a.shape[2] or not b.is_contiguous():
        raise ValueError("per-head products need contiguous heads")
    f32 = a.dtype == torch.float32
    ok = (not f32 and all(x % 8 == 0 for x in (a.stride(0), a.stride(1), out.stride(0), out.stride(1), b.shape[2], N, K))
          and a.data_ptr() % 16 == 0 and b.data_ptr() % 16 == 0 and out.data_ptr() % 16 == 0
          and (gate is None or gate.shape[1] == H or (gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0)))
    if impl == "tc" and not ok:
        raise ValueError("these sizes have no tensor-core per-head product")
    name = "vb_head_gemm" if ok and impl != "simt" else "vb_head_gemm_simt"
    args = (a.data_ptr(), a.stride(0), a.stride(1), b.data_ptr(), int(b_mn), out.data_ptr(), out.stride(0), out.stride(1),
            _lib.ptr(gate), 0 if gate is None else gate.stride(0), _gate_width(gate, H, N), T, H, K, N, tail, out.shape[2])
    if name == "vb_head_gemm":
        rc = _lib.fn(name)(*args, _lib.status_word(a.device).data_ptr(), _lib.stream())
    else:
        rc = _lib.fn(name)(*args, int(f32), _lib.stream())
    _lib.check(rc, name)


def latent_attention(q: torch.Tensor, pages: torch.Tensor, block_table: torch.Tensor, cu_q: torch.Tensor,
                     seq_lens: torch.Tensor, rank: int, *, scale: float, max_ctx: int = 0, window: int = 0,
                     sink: torch.Tensor | None = None, impl: str = "auto") -> torch.Tensor:
    """Causal attention of ragged queries in the latent space: q [T, H, width] (:func:`latent_queries`) against page rows
    [NB, BS, width], whose first ``rank`` numbers are also the values; sequences as in
    :func:`~verl_b200.ops.attention.paged_attention`, as are ``window`` and ``sink``. -> [T, H, rank].

    ``impl``: "tc" = tcgen05 kernel (bf16, rows up to 640 and ranks up to 512), "simt" = CUDA-core kernel, "auto"."""
    T, H, width = q.shape
    NB, BS, _ = pages.shape
    B = seq_lens.numel()
    if q.is_cuda:
        f32 = q.dtype == torch.float32
        tc = not f32 and bool(_lib.fn("vb_latent_decode_supported")(H, width, rank, BS))
        if impl == "tc" and not tc:
            raise ValueError(f"tensor-core latent attention does not support heads={H} width={width} rank={rank} block_size={BS}")
        out = torch.empty((T, H, rank), dtype=q.dtype, device=q.device)
        if tc and impl != "simt":
            seen = max_ctx or block_table.shape[1] * BS
            chunks = ((min(seen, window + 63) if window else seen) + 63) // 64
            splits = _lib.fn("vb_latent_decode_splits")(T, H, chunks)
            work = torch.empty(T * H * splits * (rank + 2), dtype=torch.float32, device=q.device) if splits > 1 else None
            rc = _lib.fn("vb_latent_decode")(q.data_ptr(), pages.data_ptr(), NB, block_table.data_ptr(), block_table.stride(0),
                                             cu_q.data_ptr(), seq_lens.data_ptr(), T, B, H, width, rank, BS, float(scale),
                                             window, _lib.ptr(sink), splits, out.data_ptr(), _lib.ptr(work), _lib.status_word(q.device).data_ptr(),
                                             _lib.stream())
            _lib.check(rc, "vb_latent_decode")
            return out
        rc = _lib.fn("vb_paged_attention_simt")(q.data_ptr(), q.stride(0), pages.data_ptr(), pages.data_ptr(),
                                                block_table.data_ptr(), block_table.stride(0), cu_q.data_ptr(),
                                                seq_lens.data_ptr(), T, B, H, 1, width, rank, width, BS, float(scale), window,
                                                0, 0, None, 0, 0.0, _lib.ptr(sink), None, None, None, None, 0, 0, out.data_ptr(), out.stride(0),
                                                int(f32), _lib.stream())
        _lib.check(rc, "vb_paged_attention_simt")
        return out
    out = q.new_empty((T, H, rank))
    cu, lens = cu_q.tolist(), seq_lens.tolist()
    for b in range(B):
        lo, hi, n = cu[b], cu[b + 1], lens[b]
        rows = pages[block_table[b, : (n + BS - 1) // BS].long()].reshape(-1, width)[:n].float()
        s = torch.einsum("qhd,kd->hqk", q[lo:hi].float(), rows) * scale
        out[lo:hi] = torch.einsum("hqk,kr->qhr", _masked_softmax(s, window, sink), rows[:, :rank]).to(q.dtype)
    return out


def _masked_softmax(s: torch.Tensor, window: int, sink: torch.Tensor | None) -> torch.Tensor:
    """s [H, queries, keys]: the queries are the last positions of the keys."""
    H, nq, n = s.shape
    dist = torch.arange(n - nq, n)[:, None] - torch.arange(n)[None]
    s = s.masked_fill((dist < 0) | (dist >= window if window > 0 else dist < 0), float("-inf"))
    if sink is not None:  # a key without a value
        s = torch.cat((s, sink[:, None, None].expand(H, nq, 1)), -1)
    return torch.softmax(s, -1)[..., :n]


def latent_gather(pages: torch.Tensor, block_table: torch.Tensor, ctx_cu: torch.Tensor, total: int,
                  seq_lens: torch.Tensor | None = None) -> torch.Tensor:
    """Page rows of sequences one after the other: [total, width], sequence b from row ``ctx_cu[b]``. ``seq_lens`` [B]: the last
    ``ctx_cu[b + 1] - ctx_cu[b]`` of these tokens (else the first)."""
    NB, BS, width = pages.shape
    B = ctx_cu.numel() - 1
    if pages.is_cuda:
        rows = torch.empty((total, width), dtype=pages.dtype, device=pages.device)
        rc = _lib.fn("vb_latent_gather")(pages.data_ptr(), block_table.data_ptr(), block_table.stride(0), ctx_cu.data_ptr(),
                                         _lib.ptr(seq_lens), rows.data_ptr(), total, B, width * pages.element_size(), BS, _lib.stream())
        _lib.check(rc, "vb_latent_gather")
        return rows
    out, cu = [], ctx_cu.tolist()
    for b in range(B):
        n = cu[b + 1] - cu[b]
        end = n if seq_lens is None else int(seq_lens[b])
        out.append(pages[block_table[b, : (end + BS - 1) // BS].long()].reshape(-1, width)[end - n : end])
    return torch.cat(out)


def latent_prefill(q: torch.Tensor, rot: torch.Tensor, kv: torch.Tensor, cu_q: torch.Tensor, ctx_cu: torch.Tensor, max_q: int,
                   dim: int, vdim: int, *, scale: float, gate: torch.Tensor | None, out: torch.Tensor, window: int = 0,
                   sink: torch.Tensor | None = None) -> None:
    """Causal attention of ragged queries over expanded keys and values. q [all tokens, H, dim + rot_dim]; ``rot`` [N, rot_dim]
    rotated key parts and ``kv`` [N, H x dim keys | H x vdim values | ...] of the contexts, sequence b from row ``ctx_cu[b]``;
    its queries are rows ``cu_q[b]`` to ``cu_q[b + 1]``, the last positions of its context. Writes these rows of ``out``
    [all tokens, H * vdim], times the sigmoid of ``gate`` [all tokens, H * vdim] (or [all tokens, H]: one number per head).
    ``window`` and ``sink`` as in :func:`~verl_b200.ops.attention.paged_attention`."""
    _, H, D = q.shape
    B = ctx_cu.numel() - 1
    if q.is_cuda:
        rc = _lib.fn("vb_latent_flash")(q.data_ptr(), q.stride(0), q.shape[0], rot.data_ptr(), rot.stride(0), kv.data_ptr(),
                                        kv.stride(0), kv.shape[0], cu_q.data_ptr(), ctx_cu.data_ptr(), B, max_q, H, dim, D - dim,
                                        vdim, float(scale), int(window), _lib.ptr(sink), _lib.ptr(gate),
                                        0 if gate is None else gate.stride(0), _gate_width(gate, H, vdim),
                                        out.data_ptr(), out.stride(0), _lib.status_word(q.device).data_ptr(), _lib.stream())
        _lib.check(rc, "vb_latent_flash")
        return
    cu, cc = cu_q.tolist(), ctx_cu.tolist()
    for b in range(B):
        lo, hi, n = cu[b], cu[b + 1], cc[b + 1] - cc[b]
        k, r = kv[cc[b] : cc[b + 1]].float(), rot[cc[b] : cc[b + 1]].float()
        keys = torch.cat((k[:, : H * dim].view(n, H, dim), r[:, None].expand(n, H, D - dim)), -1)
        s = torch.einsum("qhd,khd->hqk", q[lo:hi].float(), keys) * scale
        o = torch.einsum("hqk,khv->qhv", _masked_softmax(s, window, sink),
                         k[:, H * dim : H * (dim + vdim)].view(n, H, vdim)).reshape(hi - lo, -1)
        out[lo:hi] = _times_gate(o, None if gate is None else gate[lo:hi], H).to(out.dtype)
