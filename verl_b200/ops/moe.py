"""Mixture-of-experts building blocks: device-side routing layout and grouped GEMMs (one launch for all experts).

The routed tokens are sorted by expert into a buffer in which every expert's rows are padded to a multiple of 128,
so that a GEMM tile never straddles two experts; ``blk_expert`` names the expert of every 128-row block. Nothing is
read back to the host (no per-expert Python loop, no ``.tolist()``): the padded size is the static upper bound
``T * k + E * 127``. The reference leaves this to Megatron / vLLM fused-MoE kernels (grouped GEMM + permute).
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _lib
from .nn import activation, add_rmsnorm, rmsnorm_add

BLK = 128


def moe_layout(top_i: torch.Tensor, E: int):
    """top_i [T, k] expert ids -> (dest [T*k] row of every (token, slot) pair in the padded sorted buffer,
    blk_expert int32 [P / 128], expert_off int32 [E + 1] padded row offsets, P)."""
    T, k = top_i.shape
    flat = top_i.reshape(-1)
    P = ((T * k + E * (BLK - 1)) + BLK - 1) // BLK * BLK
    order = torch.argsort(flat, stable=True)
    # (torch.bincount would read its maximum back to the host: not capturable in a CUDA graph)
    counts = torch.zeros(E, dtype=torch.long, device=flat.device).scatter_add_(0, flat, torch.ones_like(flat))
    padded = (counts + BLK - 1) // BLK * BLK
    zero = torch.zeros(1, dtype=counts.dtype, device=counts.device)
    start = torch.cat([zero, counts.cumsum(0)])          # unpadded offsets
    off = torch.cat([zero, padded.cumsum(0)])            # padded offsets
    e_sorted = flat[order]
    rank_in_e = torch.arange(T * k, device=flat.device) - start[e_sorted]
    dest_sorted = off[e_sorted] + rank_in_e
    dest = torch.empty_like(dest_sorted)
    dest[order] = dest_sorted
    blk_start = torch.arange(0, P, BLK, device=flat.device)
    blk_expert = torch.searchsorted(off[1:].contiguous(), blk_start, right=True)
    blk_expert = torch.where(blk_start < off[-1], blk_expert, torch.full_like(blk_expert, -1)).to(torch.int32)
    return dest, blk_expert, off.to(torch.int32), P


def _grouped(a, b, c, M, N, K, a_mn, b_mn, accumulate, mode, E, blk_expert, expert_off):
    rc = _lib.fn("vb_grouped_gemm_bf16")(a.data_ptr(), b.data_ptr(), c.data_ptr(), M, N, K, a.stride(0), b.stride(-2),
                                         c.stride(-2), int(a_mn), int(b_mn), int(c.dtype == torch.float32), int(accumulate),
                                         mode, E, _lib.ptr(blk_expert), _lib.ptr(expert_off),
                                         _lib.status_word(a.device).data_ptr(), _lib.stream())
    _lib.check(rc, "vb_grouped_gemm_bf16")


class _GroupedLinearFn(torch.autograd.Function):
    """y[rows of e] = xs[rows of e] @ W[e]^T for all experts at once. W [E, N, K]."""

    @staticmethod
    def forward(ctx, xs, weight, blk_expert, expert_off):
        E, N, K = weight.shape
        P = xs.shape[0]
        y = torch.zeros((P, N), dtype=xs.dtype, device=xs.device)  # unused blocks stay zero
        _grouped(xs, weight, y, P, N, K, False, False, False, 1, E, blk_expert, None)
        ctx.save_for_backward(xs, weight, blk_expert, expert_off)
        return y

    @staticmethod
    def backward(ctx, dy):
        xs, weight, blk_expert, expert_off = ctx.saved_tensors
        E, N, K = weight.shape
        P = xs.shape[0]
        dy = dy.contiguous()
        dx = None
        if ctx.needs_input_grad[0]:
            dx = torch.zeros((P, K), dtype=xs.dtype, device=xs.device)
            # dX = dY . W[e]: W[e] [N, K] is the MN-major B operand (stored [contraction, out])
            _grouped(dy, weight, dx, P, K, N, False, True, False, 1, E, blk_expert, None)
        dw = None
        if ctx.needs_input_grad[1]:
            main = getattr(weight, "main_grad", None)
            acc = main if main is not None else torch.zeros((E, N, K), dtype=torch.float32, device=xs.device)
            # dW[e] += dY_e^T . X_e, contraction over the expert's (zero-padded) rows
            _grouped(dy, xs, acc, N, K, P, True, True, True, 2, E, None, expert_off)
            dw = None if main is not None else acc.to(weight.dtype)
        return dx, dw, None, None


def grouped_linear(xs: torch.Tensor, weight: torch.Tensor, blk_expert: torch.Tensor, expert_off: torch.Tensor) -> torch.Tensor:
    if not xs.is_cuda:
        E = weight.shape[0]
        y = torch.zeros(xs.shape[0], weight.shape[1], dtype=xs.dtype, device=xs.device)
        off = expert_off.tolist()
        for e in range(E):
            if off[e + 1] > off[e]:
                y[off[e] : off[e + 1]] = xs[off[e] : off[e + 1]] @ weight[e].t()
        return y
    return _GroupedLinearFn.apply(xs, weight, blk_expert, expert_off)


def moe_mlp(x: torch.Tensor, top_i: torch.Tensor, top_w: torch.Tensor, gate_up: torch.Tensor, down: torch.Tensor, swiglu,
            expert_offset: int = 0, num_experts: int | None = None):
    """Routed expert MLP. x [T, H], top_i / top_w [T, k], gate_up [E, 2I, H], down [E, H, I].

    Expert parallelism over replicated tokens: with ``num_experts`` larger than ``E`` the matrices are the experts
    ``[expert_offset, expert_offset + E)`` of the layer; pairs routed elsewhere fall into a spare bucket whose blocks
    the grouped GEMM skips, and the result is this rank's partial sum (the ranks' results add up to the layer's)."""
    T, H = x.shape
    k = top_i.shape[1]
    E = gate_up.shape[0]
    if num_experts is not None and num_experts != E:
        local = top_i - expert_offset
        local = torch.where((local >= 0) & (local < E), local, torch.full_like(local, E))
        dest, blk_expert, expert_off, P = moe_layout(local, E + 1)
        blk_expert = torch.where(blk_expert == E, torch.full_like(blk_expert, -1), blk_expert)
        top_w = torch.where(local < E, top_w, torch.zeros_like(top_w))
        expert_off = expert_off[: E + 1].contiguous()
    else:
        dest, blk_expert, expert_off, P = moe_layout(top_i, E)
    tok = torch.arange(T * k, device=x.device) // k
    xs = torch.zeros((P, H), dtype=x.dtype, device=x.device).index_copy(0, dest, x.index_select(0, tok))
    h = swiglu(grouped_linear(xs, gate_up, blk_expert, expert_off))
    out = grouped_linear(h, down, blk_expert, expert_off)
    picked = out.index_select(0, dest).view(T, k, H)
    return (picked * top_w.to(x.dtype).unsqueeze(-1)).sum(1)


# ----------------------------------------------------------------- inference: routing, experts and their sum as fused kernels
@dataclass
class Routing:
    """Experts of a step's tokens. ``idx`` / ``weight`` [T, top]: the chosen experts and their weights (fp32); ``dest`` [T, top]:
    row of the pair in the buffer sorted by expert (``rows`` of them, every expert's share padded to :data:`BLK`);
    ``blk_expert`` [rows / BLK]: expert of each block of rows (< 0: unused)."""

    idx: torch.Tensor
    weight: torch.Tensor
    dest: torch.Tensor
    blk_expert: torch.Tensor
    rows: int


@dataclass
class RoutedSum:
    """Result of a mixture in parts: rows of the sorted buffer ``out`` [rows, H], one per pair of ``routing`` (``weigh``: still to
    be multiplied with its weight), and the ``shared`` unit's result [T, H] with the logit of its gate [T] (fp32; None: a factor of
    one)."""

    out: torch.Tensor
    routing: Routing
    weigh: bool
    shared: torch.Tensor | None = None
    shared_logit: torch.Tensor | None = None


def moe_route(logits: torch.Tensor, experts: int, top: int, counters: torch.Tensor, *, score: str = "sigmoid",
              renormalize: bool = False, correction: torch.Tensor | None = None) -> Routing:
    """The ``top`` experts of every token by the fp32 ``logits`` [T, experts | ...]. ``correction`` fp32 [experts]: added to the
    scores for the choice, not for the weights. ``counters``: int32 [experts + 1], zero before and after."""
    T = logits.shape[0]
    # an expert's padding is at most BLK - 1 rows, and experts without a token have none
    rows = (T * top + min(experts, T * top) * (BLK - 1)) // BLK * BLK
    if score not in ("sigmoid", "softmax"):
        raise ValueError(f"unknown router score {score!r}")
    if logits.is_cuda:
        new = lambda n, dt=torch.int32: torch.empty(n, dtype=dt, device=logits.device)  # noqa: E731
        r = Routing(new((T, top)), new((T, top), torch.float32), new((T, top)), new(rows // BLK), rows)
        rc = _lib.fn("vb_moe_route")(logits.data_ptr(), logits.stride(0), T, experts, top, int(score == "softmax"),
                                     int(renormalize), _lib.ptr(correction), r.idx.data_ptr(), r.weight.data_ptr(), r.dest.data_ptr(),
                                     r.blk_expert.data_ptr(), rows // BLK, counters.data_ptr(), _lib.stream())
        _lib.check(rc, "vb_moe_route")
        return r
    z = logits[:, :experts]
    s = torch.sigmoid(z) if score == "sigmoid" else torch.softmax(z, -1)
    choice = s if correction is None else s + correction
    idx = torch.sort(choice, dim=-1, descending=True, stable=True).indices[:, :top]
    w = s.gather(1, idx)
    if renormalize:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    dest, blk_expert, _, P = moe_layout(idx, experts)
    return Routing(idx, w, dest.view(T, top), blk_expert, P)


def moe_experts(x: torch.Tensor, routing: Routing, first: torch.Tensor, down: torch.Tensor, act: str, *,
                weigh_input: bool) -> torch.Tensor:
    """Units of the routed pairs: rows of the sorted buffer [rows, H] (other rows undefined). x [T, H], ``down`` [E, H, ff].
    ``act`` "silu": gated linear units, ``first`` [E, 2 * ff, H] = gate | up; "gelu", "relu2": two matrices, ``first`` [E, ff, H].
    ``weigh_input``: a gated unit runs on weight * x, which is applied behind its first, linear, product."""
    if act not in ("silu", "gelu", "relu2"):
        raise ValueError(f"unknown activation of routed experts {act!r}")
    gated = act == "silu"
    if weigh_input and not gated:
        raise NotImplementedError("experts of two matrices that run on weighted inputs")
    T, H = x.shape
    top, (E, N, _) = routing.idx.shape[1], first.shape
    ff = N // 2 if gated else N
    if not x.is_cuda:
        out = torch.zeros(routing.rows, H, dtype=x.dtype)
        for e in range(E):
            t, k = (routing.idx == e).nonzero(as_tuple=True)
            gu = x[t].float() @ first[e].float().t()
            if weigh_input:
                gu = gu * routing.weight[t, k][:, None]
            h = (F.silu(gu[:, :ff]) * gu[:, ff:]).to(x.dtype) if gated else activation(gu, ff, act).to(x.dtype)
            out[routing.dest[t, k]] = (h.float() @ down[e].float().t()).to(x.dtype)
        return out
    f32, P = int(x.dtype == torch.float32), routing.rows
    new = lambda *s, dt=x.dtype: torch.empty(s, dtype=dt, device=x.device)  # noqa: E731
    xs, scale = new(P, H), new(P, dt=torch.float32)
    rc = _lib.fn("vb_moe_gather")(x.data_ptr(), x.stride(0), routing.dest.data_ptr(), routing.weight.data_ptr(), T, top, H,
                                  xs.data_ptr(), scale.data_ptr(), f32, _lib.stream())
    _lib.check(rc, "vb_moe_gather")
    gu = grouped_product(xs, first, routing.blk_expert)
    if not gated:
        return grouped_product(activation(gu, ff, act, routing.blk_expert), down, routing.blk_expert)
    h = new(P, ff)
    rc = _lib.fn("vb_silu_glu")(gu.data_ptr(), gu.stride(0), h.data_ptr(), P, ff, scale.data_ptr() if weigh_input else None,
                                routing.blk_expert.data_ptr(), f32, _lib.stream())
    _lib.check(rc, "vb_silu_glu")
    return grouped_product(h, down, routing.blk_expert)


def grouped_product(xs: torch.Tensor, weight: torch.Tensor, blk_expert: torch.Tensor) -> torch.Tensor:
    """xs [P, K] times the matrix of each block's expert, weight [E, N, K] -> [P, N] (inference; rows of unused blocks undefined).
    fp32, and sizes that the tensor cores do not take: CUDA cores."""
    (P, K), (E, N, _) = xs.shape, weight.shape
    y = torch.empty((P, N), dtype=xs.dtype, device=xs.device)
    if xs.dtype == torch.bfloat16 and K % 8 == 0:
        _grouped(xs, weight, y, P, N, K, False, False, False, 1, E, blk_expert, None)
    else:
        rc = _lib.fn("vb_grouped_gemm_simt")(xs.data_ptr(), weight.data_ptr(), y.data_ptr(), P, N, K, blk_expert.data_ptr(),
                                             int(xs.dtype == torch.float32), _lib.stream())
        _lib.check(rc, "vb_grouped_gemm_simt")
    return y


def moe_combine(parts: RoutedSum, residual: torch.Tensor, weight: torch.Tensor | None, eps: float) -> torch.Tensor:
    """Adds the mixture's sum to the fp32 ``residual`` [T, H] IN PLACE; returns rmsnorm(residual) * weight, or without a weight
    the residual, in the parts' dtype."""
    if residual.is_cuda:
        return _moe_sum(parts, residual, eps, weight)
    return add_rmsnorm(_sum_ref(parts), residual, weight, eps, parts.out.dtype)


def moe_norm_add(parts: RoutedSum, residual: torch.Tensor, weight: torch.Tensor, eps: float, *,
                 final_weight: torch.Tensor | None = None, final_scale: float = 1.0,
                 gate: torch.Tensor | None = None) -> torch.Tensor:
    """:func:`~verl_b200.ops.nn.rmsnorm_add` of the mixture's sum."""
    if residual.is_cuda:
        return _moe_sum(parts, residual, eps, final_weight, weight, gate, final_scale)
    y = rmsnorm_add(_sum_ref(parts), residual, weight, eps, final_weight=final_weight, final_scale=final_scale, gate=gate)
    return y.to(parts.out.dtype)


def _moe_sum(parts, residual, eps, weight, post=None, gate=None, scale=1.0):
    r, dtype, (T, H) = parts.routing, parts.out.dtype, residual.shape
    y = torch.empty((T, H), dtype=dtype, device=residual.device)
    sh, lg = parts.shared, parts.shared_logit
    rc = _lib.fn("vb_moe_sum")(parts.out.data_ptr(), r.dest.data_ptr(), r.weight.data_ptr() if parts.weigh else None,
                               r.idx.shape[1], _lib.ptr(sh), 0 if sh is None else sh.stride(0), _lib.ptr(lg),
                               0 if lg is None else lg.stride(0), _lib.ptr(gate), 0 if gate is None else gate.stride(0),
                               _lib.ptr(post), residual.data_ptr(), _lib.ptr(weight), float(scale), y.data_ptr(), T, H, float(eps),
                               int(dtype == torch.float32), _lib.stream())
    _lib.check(rc, "vb_moe_sum")
    return y


def _sum_ref(parts):
    r = parts.routing
    T, top = r.idx.shape
    picked = parts.out[r.dest.reshape(-1)].view(T, top, -1).float()
    d = (picked * r.weight[..., None] if parts.weigh else picked).sum(1)
    if parts.shared is not None:
        factor = 1.0 if parts.shared_logit is None else torch.sigmoid(parts.shared_logit.float())[:, None]
        d = d + parts.shared.float() * factor
    return d
