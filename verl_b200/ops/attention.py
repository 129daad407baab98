"""Attention entry points.

* :func:`attention_varlen` — causal GQA attention over packed (remove-padding) sequences for
  training and prefill. On CUDA forward and backward are this package's tcgen05 kernels (head_dim 128);
  other head dims fall back to the ``flash_attn`` library (the reference uses it for everything through HF
  ``attn_implementation=flash_attention_2``, verl/workers/fsdp_workers.py:331). CPU: per-sequence SDPA loop.
* :func:`paged_decode_attention` / :func:`kv_cache_write` — the hand-written paged-KV decode
  path of the native rollout engine.
"""

from __future__ import annotations

import torch
import torch.nn.functional as F

from . import _lib

_flash = None


def _flash_varlen():
    global _flash
    if _flash is None:
        from flash_attn import flash_attn_varlen_func  # library kernel

        _flash = flash_attn_varlen_func
    return _flash


def flash_fwd(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_seqlens: torch.Tensor, max_seqlen: int,
              causal: bool, scale: float, need_lse: bool = True, cu_seqlens_k: torch.Tensor | None = None):
    """tcgen05 forward. q [T,Hq,128], k/v [Tk,Hk,128] bf16 with unit inner strides (views of a fused qkv buffer are
    fine). ``cu_seqlens_k``: key-side boundaries when the keys are a longer stream than the queries (prefill on top
    of cached context; causal then aligns the queries with the end of the keys). ``max_seqlen`` is the longest
    query sequence. Returns (out [T,Hq,128] bf16, lse [Hq,T] fp32 or None)."""
    T, Hq, D = q.shape
    Hk = k.shape[1]
    for t in (q, k, v):
        if t.stride(2) != 1 or t.stride(1) != D or t.dtype != torch.bfloat16:
            raise ValueError("flash_fwd expects bf16 [T, H, 128] tensors with contiguous heads")
    out = torch.empty((T, Hq, D), dtype=torch.bfloat16, device=q.device)
    lse = torch.empty((Hq, T), dtype=torch.float32, device=q.device) if need_lse else None
    rc = _lib.fn("vb_flash_fwd")(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), k.stride(0), v.stride(0),
                                 cu_seqlens.data_ptr(), _lib.ptr(cu_seqlens_k), cu_seqlens.numel() - 1, T, k.shape[0],
                                 int(max_seqlen), Hq, Hk, float(scale),
                                 int(causal), out.data_ptr(), out.stride(0), _lib.ptr(lse),
                                 _lib.status_word(q.device).data_ptr(), _lib.stream())
    _lib.check(rc, "vb_flash_fwd")
    return out, lse


def flash_bwd(q, k, v, out, lse, dout, cu_seqlens, max_seqlen: int, causal: bool, scale: float):
    """tcgen05 backward: (dq [T,Hq,128], dk, dv [T,Hk,128]) from the forward's ``out`` and ``lse`` [Hq,T]."""
    T, Hq, D = q.shape
    Hk = k.shape[1]
    dout = dout if (dout.stride(2) == 1 and dout.stride(1) == D) else dout.contiguous()
    delta = torch.empty((Hq, T), dtype=torch.float32, device=q.device)
    dq = torch.empty((T, Hq, D), dtype=torch.bfloat16, device=q.device)
    dk = torch.empty((T, Hk, D), dtype=torch.bfloat16, device=q.device)
    dv = torch.empty_like(dk)
    st, stream = _lib.status_word(q.device).data_ptr(), _lib.stream()
    B = cu_seqlens.numel() - 1
    rc = _lib.fn("vb_flash_bwd_delta")(out.data_ptr(), dout.data_ptr(), out.stride(0), dout.stride(0), delta.data_ptr(), T, Hq, stream)
    _lib.check(rc, "vb_flash_bwd_delta")
    common = (q.data_ptr(), k.data_ptr(), v.data_ptr(), dout.data_ptr(), q.stride(0), k.stride(0), v.stride(0), dout.stride(0),
              cu_seqlens.data_ptr(), B, T, int(max_seqlen), Hq, Hk, float(scale), int(causal), lse.data_ptr(), delta.data_ptr())
    rc = _lib.fn("vb_flash_bwd_dq")(*common, dq.data_ptr(), dq.stride(0), st, stream)
    _lib.check(rc, "vb_flash_bwd_dq")
    rc = _lib.fn("vb_flash_bwd_dkv")(*common, dk.data_ptr(), dv.data_ptr(), dk.stride(0), st, stream)
    _lib.check(rc, "vb_flash_bwd_dkv")
    return dq, dk, dv


class _FlashVarlenFn(torch.autograd.Function):
    """Own forward and backward kernels (head_dim 128)."""

    @staticmethod
    def forward(ctx, q, k, v, cu_seqlens, max_seqlen, causal, scale):
        out, lse = flash_fwd(q, k, v, cu_seqlens, max_seqlen, causal, scale)
        ctx.save_for_backward(q, k, v, out, lse, cu_seqlens)
        ctx.max_seqlen, ctx.causal, ctx.scale = max_seqlen, causal, scale
        return out

    @staticmethod
    def backward(ctx, dout):
        q, k, v, out, lse, cu = ctx.saved_tensors
        if _BWD_IMPL == "library":
            from flash_attn.flash_attn_interface import _flash_attn_varlen_backward  # library kernel

            qc, kc, vc = q.contiguous(), k.contiguous(), v.contiguous()
            dq, dk, dv = torch.empty_like(qc), torch.empty_like(kc), torch.empty_like(vc)
            _flash_attn_varlen_backward(dout.contiguous(), qc, kc, vc, out, lse, dq, dk, dv, cu, cu, ctx.max_seqlen,
                                        ctx.max_seqlen, 0.0, ctx.scale, ctx.causal, -1, -1, 0.0, None, False, None)
            return dq, dk, dv, None, None, None, None
        dq, dk, dv = flash_bwd(q, k, v, out, lse, dout, cu, ctx.max_seqlen, ctx.causal, ctx.scale)
        return dq, dk, dv, None, None, None, None


# "native" (default) or "library": which backward the autograd wrapper uses (the library one is kept for comparisons)
_BWD_IMPL = __import__("os").environ.get("VERL_B200_ATTN_BWD", "native")


def _native_fwd_ok(q, k, v) -> bool:
    D = q.shape[-1]
    return (q.dtype == torch.bfloat16 and D == 128 and q.shape[1] % k.shape[1] == 0
            and all(t.stride(2) == 1 and t.stride(1) == D and t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0 for t in (q, k, v)))


def attention_varlen(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_seqlens: torch.Tensor, max_seqlen: int,
                     causal: bool = True, softmax_scale: float | None = None, impl: str = "auto") -> torch.Tensor:
    """q [T,Hq,D], k/v [T,Hk,D] packed; cu_seqlens int32 [B+1]. Returns [T,Hq,D].
    ``impl``: "native" forces the tcgen05 forward, "library" the flash_attn kernels, "auto" picks native when it applies."""
    D = q.shape[-1]
    scale = softmax_scale if softmax_scale is not None else D ** -0.5
    if q.is_cuda:
        native = impl != "library" and _native_fwd_ok(q, k, v)
        if impl == "native" and not native:
            raise ValueError("native attention forward needs bf16, head_dim 128 and contiguous heads")
        if native:
            if torch.is_grad_enabled() and (q.requires_grad or k.requires_grad or v.requires_grad):
                return _FlashVarlenFn.apply(q, k, v, cu_seqlens, int(max_seqlen), bool(causal), float(scale))
            return flash_fwd(q, k, v, cu_seqlens, int(max_seqlen), bool(causal), float(scale), need_lse=False)[0]
        return _flash_varlen()(q, k, v, cu_seqlens, cu_seqlens, max_seqlen, max_seqlen, softmax_scale=scale,
                               causal=causal)
    out = torch.empty_like(q)
    G = q.shape[1] // k.shape[1]
    bounds = cu_seqlens.tolist()
    for s, e in zip(bounds[:-1], bounds[1:]):
        qs = q[s:e].transpose(0, 1).unsqueeze(0)
        ks = k[s:e].repeat_interleave(G, dim=1).transpose(0, 1).unsqueeze(0)
        vs = v[s:e].repeat_interleave(G, dim=1).transpose(0, 1).unsqueeze(0)
        o = F.scaled_dot_product_attention(qs, ks, vs, is_causal=causal, scale=scale)
        out[s:e] = o.squeeze(0).transpose(0, 1)
    return out


def kv_cache_write(k: torch.Tensor, v: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor,
                   v_cache: torch.Tensor) -> None:
    """Scatter new keys/values [T,Hk,D] into the paged caches [NB,Hk,BS,D] at flat ``slots`` (int64, <0 skips)."""
    T, Hk, D = k.shape
    BS = k_cache.shape[2]
    if k.is_cuda:
        rc = _lib.fn("vb_kv_cache_write")(k.data_ptr(), v.data_ptr(), k.stride(0), v.stride(0), slots.data_ptr(),
                                          k_cache.data_ptr(), v_cache.data_ptr(), T, Hk, D, BS, _lib.stream())
        _lib.check(rc, "vb_kv_cache_write")
        return
    ok = slots >= 0
    blk, off = slots[ok] // BS, slots[ok] % BS
    k_cache[blk, :, off] = k[ok]
    v_cache[blk, :, off] = v[ok]


def decode_workspace(B: int, Hq: int, Hk: int, D: int, max_seq_len: int, device) -> tuple[int, torch.Tensor | None]:
    """Split count and fp32 scratch for :func:`paged_decode_attention` at these sizes."""
    if torch.device(device).type != "cuda":
        return 1, None
    splits = _lib.fn("vb_decode_num_splits")(B, Hk, max_seq_len)
    work = torch.empty(B * Hq * splits * (D + 2), dtype=torch.float32, device=device) if splits > 1 else None
    return splits, work


def paged_decode_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                           seq_lens: torch.Tensor, scale: float | None = None, num_splits: int = 1,
                           work: torch.Tensor | None = None, out: torch.Tensor | None = None,
                           impl: str = "auto") -> torch.Tensor:
    """One query token per sequence. q [B,Hq,D]; caches [NB,Hk,BS,D]; block_table int32 [B,max_blocks];
    seq_lens int32 [B] (including the current token, already written to the cache).

    ``impl``: "tc" = tcgen05 kernel (head_dim 128, <= 16 query heads per KV head, block size a power of two in
    8..128), "simt" = CUDA-core kernel, "auto" = "tc" wherever it applies."""
    B, Hq, D = q.shape
    Hk, BS = k_cache.shape[1], k_cache.shape[2]
    scale = scale if scale is not None else D ** -0.5
    if out is None:
        out = torch.empty_like(q)
    if q.is_cuda:
        if num_splits > 1 and work is None:
            work = torch.empty(B * Hq * num_splits * (D + 2), dtype=torch.float32, device=q.device)
        tc_ok = bool(_lib.fn("vb_paged_decode_tc_supported")(Hq, Hk, D, BS)) and k_cache.is_contiguous() and v_cache.is_contiguous()
        if impl == "tc" and not tc_ok:
            raise ValueError(f"tensor-core decode does not support Hq={Hq} Hk={Hk} D={D} block_size={BS}")
        if tc_ok and impl != "simt":
            rc = _lib.fn("vb_paged_decode_tc")(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(),
                                               k_cache.shape[0], block_table.data_ptr(), block_table.stride(0),
                                               seq_lens.data_ptr(), B, Hq, Hk, BS, scale, num_splits, out.data_ptr(),
                                               out.stride(0), _lib.ptr(work), _lib.status_word(q.device).data_ptr(),
                                               _lib.stream())
            _lib.check(rc, "vb_paged_decode_tc")
            return out
        rc = _lib.fn("vb_paged_decode")(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(),
                                        block_table.data_ptr(), block_table.stride(0), seq_lens.data_ptr(), B, Hq, Hk,
                                        D, BS, scale, num_splits, out.data_ptr(), out.stride(0), _lib.ptr(work),
                                        _lib.stream())
        _lib.check(rc, "vb_paged_decode")
        return out
    G = Hq // Hk
    for b in range(B):
        L = int(seq_lens[b])
        nb = (L + BS - 1) // BS
        blocks = block_table[b, :nb].long()
        kk = k_cache[blocks].permute(1, 0, 2, 3).reshape(Hk, -1, D)[:, :L].float()
        vv = v_cache[blocks].permute(1, 0, 2, 3).reshape(Hk, -1, D)[:, :L].float()
        qq = q[b].float().reshape(Hk, G, D)
        s = torch.einsum("hgd,hld->hgl", qq, kk) * scale
        out[b] = torch.einsum("hgl,hld->hgd", torch.softmax(s, -1), vv).reshape(Hq, D).to(q.dtype)
    return out


# ----------------- paged attention of layer-list decoders (windows, chunks, kept keys, distance bias, soft cap, sink, gate)
def qk_norm_kv_write(qkv: torch.Tensor, q_weight: torch.Tensor | None, k_weight: torch.Tensor | None, slots: torch.Tensor,
                     k_cache: torch.Tensor, v_cache: torch.Tensor, heads: int, eps: float, *,
                     q_temp: tuple | None = None, positions: torch.Tensor | None = None) -> torch.Tensor:
    """``qkv`` [T, q | k | v | padding]: RMS norm of q and of k over the whole projection (all heads at once; no weights =
    no norm), k and v to their places in the paged caches [NB, Hk, BS, D] / [NB, Hk, BS, Dv] (slot < 0: no write).
    ``q_temp`` (coef, every): the query at position p is multiplied by 1 + coef * ln(floor((p + 1) / every) + 1). Returns q [T, heads, D], a view of ``qkv`` (normalised in place on CUDA)."""
    _, Hk, BS, D = k_cache.shape
    Dv = v_cache.shape[3]
    T, nq, nk = qkv.shape[0], heads * D, Hk * D
    if qkv.is_cuda:
        rc = _lib.fn("vb_qk_norm_kv_write")(qkv.data_ptr(), qkv.stride(0), _lib.ptr(q_weight), _lib.ptr(k_weight),
                                            slots.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), T, heads, Hk, D, Dv, BS,
                                            float(eps), None if q_temp is None else positions.data_ptr(),
                                            *(q_temp or (0.0, 1.0)), int(qkv.dtype == torch.float32), _lib.stream())
        _lib.check(rc, "vb_qk_norm_kv_write")
        return qkv[:, :nq].view(T, heads, D)
    from .nn import _rmsnorm_ref

    q, k, v = qkv[:, :nq], qkv[:, nq : nq + nk], qkv[:, nq + nk : nq + nk + Hk * Dv]
    if q_weight is not None:
        q, k = _rmsnorm_ref(q.float(), q_weight.float(), eps), _rmsnorm_ref(k, k_weight, eps)
    if q_temp is not None:
        q = q.float() * (1 + q_temp[0] * torch.log(torch.floor((positions.double() + 1) / q_temp[1]) + 1)).float()[:, None]
    q = q.to(qkv.dtype)
    kv_cache_write(k.reshape(T, Hk, D), v.reshape(T, Hk, Dv), slots, k_cache, v_cache)
    return q.reshape(T, heads, D)


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, freqs: torch.Tensor, interleaved: bool,
                 amplitude: float = 1.0) -> torch.Tensor:
    """fp32 rotary positions on the first ``2 * len(freqs)`` of the last dimension of x [T, ..., D] (reference form)."""
    x, n = x.float(), freqs.numel()
    a = (positions.float()[:, None] * freqs).view([x.shape[0]] + [1] * (x.dim() - 2) + [n])
    c, s = a.cos() * amplitude, a.sin() * amplitude
    r = x[..., : 2 * n]
    u, v = (r[..., 0::2], r[..., 1::2]) if interleaved else (r[..., :n], r[..., n:])
    u, v = u * c - v * s, v * c + u * s
    r = torch.stack((u, v), -1).flatten(-2) if interleaved else torch.cat((u, v), -1)
    return torch.cat((r, x[..., 2 * n :]), -1)


def head_norm_rope_kv_write(qkv: torch.Tensor, q_weight: torch.Tensor | None, k_weight: torch.Tensor | None,
                            freqs: torch.Tensor | None, positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor,
                            v_cache: torch.Tensor, heads: int, eps: float, *, interleaved: bool,
                            amplitude: float = 1.0, key_values: bool = False) -> torch.Tensor:
    """``qkv`` [T, q | k | v | ...]: RMS norm of every q and k head (weights [D] shared by the heads; None = no norm), rotary
    positions with the angles ``positions * freqs`` (fp32; None = none) on the first ``2 * len(freqs)`` dimensions, k and v
    to their places in the paged caches [NB, Hk, BS, D] / [NB, Hk, BS, Dv] (slot < 0: no write). ``key_values``: there is no v,
    the keys' projection goes to the value cache as it is. Returns q [T, heads, D], a view of ``qkv`` (changed in place on CUDA)."""
    _, Hk, BS, D = k_cache.shape
    Dv = v_cache.shape[3]
    T, nq, nk = qkv.shape[0], heads * D, Hk * D
    if key_values and Dv != D:
        raise ValueError(f"values of {Dv} that are the keys of {D}")
    if qkv.is_cuda:
        rc = _lib.fn("vb_head_norm_rope_kv_write")(
            qkv.data_ptr(), qkv.stride(0), _lib.ptr(q_weight), _lib.ptr(k_weight), _lib.ptr(freqs),
            0 if freqs is None else freqs.numel(), int(interleaved), float(amplitude), positions.data_ptr(), slots.data_ptr(),
            k_cache.data_ptr(), v_cache.data_ptr(), T, heads, Hk, D, Dv, BS, int(key_values), float(eps),
            int(qkv.dtype == torch.float32), _lib.stream())
        _lib.check(rc, "vb_head_norm_rope_kv_write")
        return qkv[:, :nq].view(T, heads, D)
    from .nn import _rmsnorm_ref

    q, k = qkv[:, :nq].view(T, heads, D), qkv[:, nq : nq + nk].view(T, Hk, D)
    v = k if key_values else qkv[:, nq + nk : nq + nk + Hk * Dv]
    if q_weight is not None:
        q, k = (_rmsnorm_ref(x.float(), w.float(), eps) for x, w in ((q, q_weight), (k, k_weight)))
    if freqs is not None:
        q, k = (rotate_pairs(x, positions, freqs, interleaved, amplitude) for x in (q, k))
    kv_cache_write(k.to(qkv.dtype), v.reshape(T, Hk, Dv), slots, k_cache, v_cache)
    return q.to(qkv.dtype)


def paged_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                    cu_q: torch.Tensor, seq_lens: torch.Tensor, max_q: int, *, scale: float, window: int = 0,
                    keep_first: int = 0, bias: torch.Tensor | None = None, max_ctx: int = 0, chunk: int = 0,
                    softcap: float = 0.0, sink: torch.Tensor | None = None, gate: torch.Tensor | None = None,
                    shift: torch.Tensor | None = None, log_bias: tuple | None = None, impl: str = "auto") -> torch.Tensor:
    """Causal attention of ragged queries (the last ``cu_q[b + 1] - cu_q[b]`` positions of every sequence) over the paged
    cache, which holds the new tokens already. q [T, Hq, D]; caches [NB, Hk, BS, D] / [NB, Hk, BS, Dv]; ``seq_lens``
    [B] = tokens of each sequence including the new ones. ``window`` > 0: position i sees j <= i with i - j < window or
    j < keep_first. ``bias`` fp32 [Hq, L]: ``bias[h, min(i - j, L - 1)]`` is added to the scaled score. ``chunk`` > 0:
    position i sees j <= i with i // chunk == j // chunk (not together with a window). ``softcap`` > 0: scores become
    ``softcap * tanh(score / softcap)`` (without a bias). ``sink`` fp32 [Hq]: exp(sink[h]) joins the softmax denominator.
    ``shift`` fp32 [Hq]: no softmax, a key weighs sigmoid(score + shift[h]) (without bias, soft cap and sink). ``log_bias`` = (r1,
    r2), fp32 [Hq] each, only then: r1[h] * ln(1 + r2[h] * (i - j)) is taken off the scaled score. ``gate`` [T, Hq * Dv] or
    [T, Hq]: the result is multiplied with its sigmoid. ``max_ctx``: bound of ``seq_lens``. -> [T, Hq * Dv].

    ``impl``: "tc" = tcgen05 kernels (bf16, head sizes up to 128 in multiples of 8, block size a power of two in 8..128;
    one token per sequence: up to 8 query heads per KV head), "simt" = CUDA-core kernel, "auto" = "tc" where it applies."""
    T, Hq, D = q.shape
    Hk, BS, Dv = k_cache.shape[1], k_cache.shape[2], v_cache.shape[3]
    B = seq_lens.numel()
    out = torch.empty((T, Hq * Dv), dtype=q.dtype, device=q.device)
    if (chunk > 0 and window > 0) or (softcap > 0 and bias is not None):
        raise ValueError("paged_attention: chunk goes without window, and softcap without bias")
    if (shift is not None and (bias is not None or softcap > 0 or sink is not None)) or (log_bias is not None and shift is None):
        raise ValueError("paged_attention: sigmoid weights go without bias table, soft cap and sink, a log bias only with them")
    gate_w = 0 if gate is None else gate.shape[1] // Hq  # numbers of the gate per head
    if gate is not None and gate.shape[1] not in (Hq, Hq * Dv):
        raise ValueError(f"paged_attention: a gate of {gate.shape[1]} numbers for {Hq} heads of {Dv}")
    if q.is_cuda:
        f32 = q.dtype == torch.float32
        L = 0 if bias is None else bias.shape[1]
        if max_q == 1:
            tc = _lib.fn("vb_paged_decode_window_supported")(Hq, Hk, D, Dv, BS)
        else:
            tc = _lib.fn("vb_paged_flash_supported")(Hq, Hk, D, Dv, BS, L)
        tc = bool(tc) and not f32 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0
        if gate is not None and gate_w > 1:
            tc = tc and gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0
        if impl == "tc" and not tc:
            raise ValueError(f"tensor-core attention does not support Hq={Hq} Hk={Hk} D={D} Dv={Dv} block_size={BS}")
        args = (q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr())
        table = (block_table.data_ptr(), block_table.stride(0))
        r1, r2 = log_bias or (None, None)
        mask = (float(scale), window, keep_first, chunk, _lib.ptr(bias), L, float(softcap), _lib.ptr(sink), _lib.ptr(shift),
                _lib.ptr(r1), _lib.ptr(r2), _lib.ptr(gate), 0 if gate is None else gate.stride(0), gate_w)
        dst = (out.data_ptr(), out.stride(0))
        if tc and impl != "simt" and max_q == 1:
            seen = max_ctx or block_table.shape[1] * BS
            if window > 0:
                seen = min(seen, window + keep_first + 128)
            elif chunk > 0:
                seen = min(seen, chunk + 128)
            # split the keys only as far as all pieces run at once (two CTAs per SM): windows leave few chunks to walk
            sms = torch.cuda.get_device_properties(q.device).multi_processor_count
            splits = max(1, min(2 * sms // (B * Hk), (seen + 127) // 128, 16))
            work = torch.empty(B * Hq * splits * (Dv + 2), dtype=torch.float32, device=q.device) if splits > 1 else None
            rc = _lib.fn("vb_paged_decode_window")(*args, k_cache.shape[0], *table, seq_lens.data_ptr(), B, Hq, Hk, D, Dv, BS,
                                                   *mask, splits, *dst, _lib.ptr(work),
                                                   _lib.status_word(q.device).data_ptr(), _lib.stream())
        elif tc and impl != "simt":
            rc = _lib.fn("vb_paged_flash")(*args, k_cache.shape[0], *table, cu_q.data_ptr(), seq_lens.data_ptr(), T, B, max_q,
                                           Hq, Hk, D, Dv, BS, *mask, *dst, _lib.status_word(q.device).data_ptr(),
                                           _lib.stream())
        else:
            rc = _lib.fn("vb_paged_attention_simt")(*args, *table, cu_q.data_ptr(), seq_lens.data_ptr(), T, B, Hq, Hk, D, Dv, Dv, BS,
                                                    *mask, *dst, int(f32), _lib.stream())
        _lib.check(rc, "paged_attention")
        return out
    G = Hq // Hk
    cu, lens = cu_q.tolist(), seq_lens.tolist()
    for b in range(B):
        lo, hi, n = cu[b], cu[b + 1], lens[b]
        if hi == lo:
            continue
        blocks = block_table[b, : (n + BS - 1) // BS].long()
        kk = k_cache[blocks].permute(1, 0, 2, 3).reshape(Hk, -1, D)[:, :n].float().repeat_interleave(G, 0)
        vv = v_cache[blocks].permute(1, 0, 2, 3).reshape(Hk, -1, Dv)[:, :n].float().repeat_interleave(G, 0)
        s = torch.einsum("qhd,hkd->hqk", q[lo:hi].float(), kk) * scale
        dist = torch.arange(n - (hi - lo), n, device=q.device)[:, None] - torch.arange(n, device=q.device)[None]
        seen = dist >= 0
        if window > 0:
            seen &= (dist < window) | (torch.arange(n, device=q.device)[None] < keep_first)
        if chunk > 0:
            at = torch.arange(n, device=q.device) // chunk
            seen &= at[n - (hi - lo) :, None] == at[None]
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        if bias is not None:
            s = s + bias[:, dist.clamp(0, bias.shape[1] - 1)]
        if shift is not None:
            if log_bias is not None:
                r1, r2 = (r[:, None, None] for r in log_bias)
                s = s - r1 * torch.log1p(r2 * dist.clamp(min=0))
            w = torch.sigmoid(s + shift[:, None, None]).masked_fill(~seen, 0.0)
            out[lo:hi] = _head_gate(torch.einsum("hqk,hkd->qhd", w, vv), None if gate is None else gate[lo:hi]).to(q.dtype)
            continue
        s = s.masked_fill(~seen, float("-inf"))
        if sink is not None:  # a key without a value
            s = torch.cat((s, sink[:, None, None].expand(Hq, hi - lo, 1)), -1)
        o = torch.einsum("hqk,hkd->qhd", torch.softmax(s, -1)[..., :n], vv)
        out[lo:hi] = _head_gate(o, None if gate is None else gate[lo:hi]).to(q.dtype)
    return out


def _head_gate(o: torch.Tensor, gate: torch.Tensor | None) -> torch.Tensor:
    """o [T, H, D] times the sigmoid of ``gate`` [T, H * D] or [T, H] -> [T, H * D]."""
    if gate is not None:
        o = o * torch.sigmoid(gate.float().view(o.shape[0], o.shape[1], -1))
    return o.reshape(o.shape[0], -1)
