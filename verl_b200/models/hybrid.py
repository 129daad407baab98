"""Decoders described layer by layer (``ModelConfig.layer_specs``): every layer has its own mixer, attention over the paged
KV cache, latent attention over pages of latents, a gated delta rule, gated linear attention or a gated linear recurrent unit
with per-sequence state, and an optional feed-forward or mixture of them.

Served by the rollout engine like the homogeneous stacks of :mod:`.transformer`; there is no training path. The residual
stream is fp32 and every norm is fused with the residual add beside it. Designs that norm what a sublayer reads:

    embedding * scale -> [ add + norm1 -> fused input projection -> mixer -> output projection
                           -> add + norm2 -> gate|up -> GLU -> down ] ... -> add + final norm -> head

Designs that norm what a sublayer puts out (the last norm + add also computes the final norm):

    embedding * scale -> [ fused input projection -> mixer -> output projection -> norm1 + add
                           -> gate|up -> GLU -> down -> norm2 + add ] ... -> head

Designs that norm both, with a gate on what a sublayer puts out (its projection is part of the sublayer's first matrix):

    embedding + position -> [ norm1 -> fused input projection -> mixer -> output projection -> gate, norm1b, add + norm2
                              -> up -> activation -> down -> gate, norm2b, add + next norm ] ... -> head

Layers with an input of their own per token read the stream behind the feed-forward as it is, and their normed output is added
together with the next layer's norm1 (or the final norm):

    [ ... add + copy -> gate -> gelu * side embedding -> out -> norm + add + next norm ]
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Callable, Optional

import torch
import torch.nn as nn

from .. import ops
from .config import ModelConfig
from .layer_specs import (AttentionSpec, DeltaSpec, GlaSpec, GluSpec, LatentSpec, LayerSpec, LruSpec, MlpSpec, MoeSpec,
                          distance_buckets, weight_owner)
from .transformer import Linear, RMSNormWeight


# Latent attention: portions of up to LATENT_SHORT tokens attend in the latent space (more arithmetic per key, no expansion);
# longer ones expand keys and values of up to LATENT_GROUP context tokens at a time (or of one longer sequence).
LATENT_SHORT, LATENT_GROUP = 32, 1 << 17


def pad8(n: int) -> int:
    """Rows of a fused projection: a multiple of 8 keeps the rows of its output 16-byte aligned."""
    return (n + 7) // 8 * 8


@dataclass
class LatentPlan:
    """How latent-attention layers run a step. The leading ``short_seqs`` sequences (``short_rows`` token rows, few new tokens
    each) attend in the latent space, straight from the pages. The others get the keys and values of their whole context
    expanded, group by group: (first sequence, end, ctx_cu = int32 [n + 1] boundaries of the contexts, their total, longest
    portion). ``windowed``: the same for layers with a window, by its size: a context is what the window reaches."""

    short_seqs: int
    short_rows: int
    groups: tuple = ()
    windowed: dict = field(default_factory=dict)

    def groups_of(self, window: int) -> tuple:
        return self.windowed[window] if window else self.groups


@dataclass
class RaggedBatch:
    """One step: the new tokens of B sequences, described for the cache and state (all int32 except ``slots`` and
    ``positions``, int64)."""

    cu_q: torch.Tensor         # [B + 1] boundaries of the new tokens
    max_q: int
    seq_lens: torch.Tensor     # [B] tokens of each sequence including the new ones
    slots: torch.Tensor        # [T] cache place of each token (page * block_size + offset; < 0: padding)
    block_table: torch.Tensor  # [B, max_blocks]
    state_slots: torch.Tensor  # [B] recurrent-state slot (< 0: padding)
    max_ctx: int = 0           # longest sequence a replay of this step may see
    positions: Optional[torch.Tensor] = None  # [T] position of each token
    latent: Optional[LatentPlan] = None
    singles: int = 0           # leading sequences with one new token each


class StateCache:
    """Cache of a layer-list model: K / V pages per attention layer, pages of latents and rotated keys per latent-attention
    layer, fp32 state (and a convolution ring where the layer convolves) per recurrent layer."""

    def __init__(self, cfg: ModelConfig, num_blocks: int, block_size: int, num_slots: int, dtype, device):
        self.layers: list[tuple] = []
        for spec in cfg.layer_specs:
            m = spec.mixer
            if spec.kind == "attention":
                self.layers.append(tuple(torch.zeros((num_blocks, m.kv_heads, block_size, d), dtype=dtype, device=device)
                                         for d in (m.dim, m.vdim)))
            elif spec.kind == "latent_attention":
                self.layers.append((torch.zeros((num_blocks, block_size, ops.latent_width(m.latent_size)), dtype=dtype, device=device),))
            else:
                channels, state = self._state(spec)
                ring = (torch.zeros((num_slots, m.conv, channels), dtype=dtype, device=device),) if channels else ()
                self.layers.append((*ring, torch.zeros((num_slots, *state), dtype=torch.float32, device=device)))

    @staticmethod
    def _state(spec) -> tuple:
        """Convolved channels and shape of the state of a recurrent layer."""
        m = spec.mixer
        if spec.kind == "rglru":
            return m.width, (m.width,)
        return 0 if spec.kind == "gla" else m.channels, (m.heads, m.vdim, m.dim)

    @staticmethod
    def page_bytes(cfg: ModelConfig, block_size: int, itemsize: int) -> int:
        per_token = {"attention": lambda m: m.kv_heads * (m.dim + m.vdim), "latent_attention": lambda m: ops.latent_width(m.latent_size)}
        return sum(per_token[s.kind](s.mixer) for s in cfg.layer_specs if s.kind in per_token) * block_size * itemsize

    @staticmethod
    def slot_bytes(cfg: ModelConfig, itemsize: int) -> int:
        total = 0
        for s in cfg.layer_specs:
            if s.kind in ("delta", "gla", "rglru"):
                channels, state = StateCache._state(s)
                total += (s.mixer.conv * channels * itemsize if channels else 0) + 4 * math.prod(state)
        return total


def rotary_frequencies(module: nn.Module, spec, device) -> None:
    """The rotation's frequencies as the module's fp32 buffer ``rot_freqs``."""
    module.register_buffer("rot_freqs", torch.tensor(spec.frequencies(), dtype=torch.float32, device=device), persistent=False)


class Sublayer(nn.Module):
    """A mixer or feed-forward: its spec, and the rows of a residual gate (0: none) behind the ``own`` rows of its first matrix,
    from a multiple of 8 on."""

    def __init__(self, cfg: ModelConfig, spec, own: int):
        super().__init__()
        self.spec, self.eps = spec, cfg.rms_norm_eps
        self.gate_rows = cfg.hidden_size if cfg.design.residual_gate else 0
        self.own = own

    def first_matrix(self, cfg: ModelConfig, bias: bool, dtype, device) -> Linear:
        rows = pad8(self.own) + pad8(self.gate_rows) if self.gate_rows else pad8(self.own)
        return Linear(cfg.hidden_size, rows, bias or self.gate_rows > 0, dtype, device)

    def residual_gate(self, proj):
        """Logits of the residual gate out of the first matrix' result, or None."""
        lo = pad8(self.own)
        return proj[:, lo : lo + self.gate_rows] if self.gate_rows else None


class Mixer(Sublayer):
    """``forward(x, batch, cache, mm)``: (result, logits of its residual gate or None)."""

    def refresh(self):
        """Derived tables, after the weights have changed."""


class AttentionMixer(Mixer):
    def __init__(self, cfg: ModelConfig, spec: AttentionSpec, dtype, device):
        super().__init__(cfg, spec, spec.proj_size)
        self.qkv_proj = self.first_matrix(cfg, spec.qkv_bias, dtype, device)
        self.o_proj = Linear(spec.out_size, cfg.hidden_size, False, dtype, device)
        if spec.qk_norm:
            self.q_norm, self.k_norm = (RMSNormWeight(n, dtype, device) for n in spec.norm_sizes)
        if spec.sink:
            self.sink = nn.Parameter(torch.zeros(spec.heads, dtype=torch.float32, device=device))
        for n, on in (("r1", spec.log_bias), ("r2", spec.log_bias), ("shift", spec.weighting == "sigmoid")):
            if on:
                setattr(self, n, nn.Parameter(torch.zeros(spec.heads, dtype=torch.float32, device=device)))
        if spec.rotary is not None:
            rotary_frequencies(self, spec.rotary, device)
        if spec.bias_rows:
            self.rel = nn.Parameter(torch.zeros(spec.bias_rows, spec.heads, dtype=torch.float32, device=device))
            buckets = torch.tensor(distance_buckets(spec.bias_rows, spec.bias_max), dtype=torch.long, device=device)
            self.register_buffer("buckets", buckets, persistent=False)
            self.register_buffer("bias", torch.zeros(spec.heads, len(buckets), dtype=torch.float32, device=device),
                                 persistent=False)

    @torch.no_grad()
    def refresh(self):
        """Per-distance bias [heads, distances] from the learned table (call when the weights have changed)."""
        if self.spec.bias_rows:
            self.bias.copy_(self.rel.t()[:, self.buckets])

    def forward(self, x, batch: RaggedBatch, cache, mm: Callable):
        s = self.spec
        norms = (self.q_norm.weight, self.k_norm.weight) if s.qk_norm else (None, None)
        qkv = mm(x, self.qkv_proj.weight, self.qkv_proj.bias)
        if s.rotary is None and (s.qk_norm == "projection" or s.q_temp is not None):
            if s.qk_norm == "head":
                raise NotImplementedError("a query temperature after a norm per head")
            q = ops.qk_norm_kv_write(qkv, *norms, batch.slots, cache[0], cache[1], s.heads, self.eps, q_temp=s.q_temp,
                                     positions=batch.positions)
        elif s.qk_norm != "projection" and s.q_temp is None:
            q = ops.head_norm_rope_kv_write(qkv, *norms, self.rot_freqs if s.rotary else None, batch.positions, batch.slots,
                                            cache[0], cache[1], s.heads, self.eps,
                                            interleaved=s.rotary is not None and s.rotary.interleaved,
                                            amplitude=s.rotary.amplitude if s.rotary else 1.0, key_values=s.key_values)
        else:
            raise NotImplementedError("rotary positions after a norm over the whole projection, or with a query temperature")
        lo = s.q_size + s.k_size + s.v_size
        o = ops.paged_attention(q, cache[0], cache[1], batch.block_table, batch.cu_q, batch.seq_lens, batch.max_q,
                                scale=s.scale, window=s.window, keep_first=s.keep_first,
                                bias=self.bias if s.bias_rows else None, max_ctx=batch.max_ctx, chunk=s.chunk,
                                softcap=s.softcap, sink=self.sink if s.sink else None,
                                gate=qkv[:, lo : lo + s.gate_size] if s.gate else None,
                                shift=self.shift if s.weighting == "sigmoid" else None,
                                log_bias=(self.r1, self.r2) if s.log_bias else None)
        return mm(o, self.o_proj.weight), self.residual_gate(qkv)


class LatentMixer(Mixer):
    def __init__(self, cfg: ModelConfig, spec: LatentSpec, dtype, device):
        super().__init__(cfg, spec, spec.proj_size)
        self.in_proj = self.first_matrix(cfg, False, dtype, device)
        self.kv_norm = RMSNormWeight(spec.kv_rank, dtype, device)
        self.kv_up_proj = Linear(spec.kv_rank, pad8(spec.up_size), False, dtype, device)
        self.o_proj = Linear(spec.out_size, cfg.hidden_size, False, dtype, device)
        if spec.q_rank:
            self.q_latent_norm = RMSNormWeight(spec.q_rank, dtype, device)
            self.q_up_proj = Linear(spec.q_rank, pad8(spec.q_size), False, dtype, device)
        if spec.sink:
            self.sink = nn.Parameter(torch.zeros(spec.heads, dtype=torch.float32, device=device))
        rotary_frequencies(self, spec.rotary, device)

    def forward(self, x, batch: RaggedBatch, cache, mm: Callable):
        s, pages, plan = self.spec, cache[0], batch.latent
        T = x.shape[0]
        proj = mm(x, self.in_proj.weight, self.in_proj.bias)
        rot = dict(amplitude=s.rotary.amplitude, interleaved=s.rotary.interleaved)
        ops.latent_rope_write(proj, self.kv_norm.weight, self.rot_freqs, batch.positions, batch.slots, pages,
                              0 if s.q_rank else s.heads, s.dim, s.rot_dim, s.kv_rank, self.eps, **rot, q_rank=s.q_rank,
                              q_norm_w=self.q_latent_norm.weight if s.q_rank else None)
        q = proj
        if s.q_rank:
            q = mm(proj[:, : s.q_rank], self.q_up_proj.weight)
            ops.rotate_tails(q, self.rot_freqs, batch.positions, s.heads, s.dim, s.rot_dim, **rot)
        q = q[:, : s.q_size].view(T, s.heads, s.dim + s.rot_dim)
        lo = s.q_in + s.latent_size
        gate = proj[:, lo : lo + s.gate_size] if s.gate else None
        sink = self.sink if s.sink else None
        out = torch.empty((T, s.out_size), dtype=x.dtype, device=x.device)
        up = self.kv_up_proj.weight
        uk = up[: s.heads * s.dim].view(s.heads, s.dim, s.kv_rank)
        uv = up[s.heads * s.dim : s.up_size].view(s.heads, s.vdim, s.kv_rank)
        n, B = plan.short_rows, plan.short_seqs
        if n:  # scores and weighted sums over the latents themselves: W_uk moves to the queries, W_uv behind the sum
            lat = ops.latent_attention(ops.latent_queries(q[:n], uk), pages, batch.block_table[:B], batch.cu_q[: B + 1],
                                       batch.seq_lens[:B], s.kv_rank, scale=s.scale, max_ctx=batch.max_ctx, window=s.window,
                                       sink=sink)
            ops.latent_values(lat, uv, None if gate is None else gate[:n], out[:n])
        for b0, b1, ctx_cu, total, max_q in plan.groups_of(s.window):
            rows = ops.latent_gather(pages, batch.block_table[b0:b1], ctx_cu, total, batch.seq_lens[b0:b1])
            kv = mm(rows[:, : s.kv_rank], up)
            ops.latent_prefill(q, rows[:, s.kv_rank : s.latent_size], kv, batch.cu_q[b0 : b1 + 1], ctx_cu, max_q, s.dim,
                               s.vdim, scale=s.scale, gate=gate, out=out, window=s.window, sink=sink)
        return mm(out, self.o_proj.weight), self.residual_gate(proj)


class DeltaMixer(Mixer):
    def __init__(self, cfg: ModelConfig, spec: DeltaSpec, dtype, device):
        super().__init__(cfg, spec, spec.proj_size)
        self.in_proj = self.first_matrix(cfg, False, dtype, device)
        self.conv = nn.Parameter(torch.zeros(spec.channels, spec.conv, dtype=dtype, device=device))
        self.A_log = nn.Parameter(torch.zeros(spec.heads, dtype=torch.float32, device=device))
        self.dt_bias = nn.Parameter(torch.zeros(spec.heads, dtype=torch.float32, device=device))
        self.norm = RMSNormWeight(spec.vdim, dtype, device)
        self.o_proj = Linear(spec.out_size, cfg.hidden_size, False, dtype, device)

    def reset_parameters(self, generator=None):
        with torch.no_grad():
            dev = self.conv.device
            self.conv.copy_(torch.empty(self.conv.shape, device=dev).normal_(0.0, self.spec.conv ** -0.5, generator=generator))
            self.A_log.copy_(torch.empty(self.spec.heads, device=dev).uniform_(1.0, 8.0, generator=generator).log())
            self.dt_bias.copy_(torch.empty(self.spec.heads, device=dev).uniform_(-5.0, -2.0, generator=generator))

    def forward(self, x, batch: RaggedBatch, cache, mm: Callable):
        s = self.spec
        proj = mm(x, self.in_proj.weight, self.in_proj.bias)
        o = ops.delta_rule(proj, self.conv, self.A_log, self.dt_bias, self.norm.weight, cache[0], cache[1], batch.cu_q,
                           batch.seq_lens, batch.state_slots, batch.max_q, s.heads, s.kv_heads, s.dim, s.vdim, self.eps)
        return mm(o, self.o_proj.weight), self.residual_gate(proj)


class GlaMixer(Mixer):
    def __init__(self, cfg: ModelConfig, spec: GlaSpec, dtype, device):
        super().__init__(cfg, spec, spec.proj_size)
        self.in_proj = self.first_matrix(cfg, False, dtype, device)
        self.decay_w = nn.Parameter(torch.zeros(spec.qk_size, spec.rank, dtype=dtype, device=device))
        self.decay_b = nn.Parameter(torch.zeros(spec.qk_size, dtype=torch.float32, device=device))
        self.norm = RMSNormWeight(spec.vdim, dtype, device)
        self.o_proj = Linear(spec.out_size, cfg.hidden_size, False, dtype, device)

    def reset_parameters(self, generator=None):
        with torch.no_grad():
            dev, n = self.decay_w.device, max(self.spec.rank, 1)
            self.decay_w.copy_(torch.empty(self.decay_w.shape, device=dev).normal_(0.0, n ** -0.5, generator=generator))
            self.decay_b.copy_(torch.empty(self.decay_b.shape, device=dev).uniform_(0.0, 4.0, generator=generator))

    def forward(self, x, batch: RaggedBatch, cache, mm: Callable):
        s = self.spec
        proj = mm(x, self.in_proj.weight, self.in_proj.bias)
        o = ops.gated_linear_attention(proj, self.decay_w, self.decay_b, self.norm.weight, cache[0], batch.cu_q, batch.seq_lens,
                                       batch.state_slots, batch.max_q, s.heads, s.dim, s.vdim, s.tau, self.eps,
                                       singles=batch.singles)
        return mm(o, self.o_proj.weight), self.residual_gate(proj)


class LruMixer(Mixer):
    def __init__(self, cfg: ModelConfig, spec: LruSpec, dtype, device):
        super().__init__(cfg, spec, spec.proj_size)
        n = spec.block_size
        self.in_proj = self.first_matrix(cfg, True, dtype, device)
        self.conv_w = nn.Parameter(torch.zeros(spec.width, spec.conv, dtype=dtype, device=device))
        self.conv_b = nn.Parameter(torch.zeros(spec.width, dtype=dtype, device=device))
        self.gates = nn.Parameter(torch.zeros(2 * spec.blocks, n, n, dtype=dtype, device=device))  # decay | input
        self.gates_b = nn.Parameter(torch.zeros(2 * spec.blocks, n, dtype=torch.float32, device=device))
        self.lam = nn.Parameter(torch.zeros(spec.width, dtype=torch.float32, device=device))
        self.o_proj = Linear(spec.out_size, cfg.hidden_size, False, dtype, device)

    def reset_parameters(self, generator=None):
        with torch.no_grad():
            for w, fan in ((self.conv_w, self.spec.conv), (self.gates, self.spec.block_size)):
                w.copy_(torch.empty(w.shape, device=w.device).normal_(0.0, fan ** -0.5, generator=generator))
            # decays (at a gate of one) between 0.9 and 0.999
            a = torch.empty(self.spec.width, device=self.lam.device).uniform_(0.9, 0.999, generator=generator)
            self.lam.copy_(torch.log(torch.expm1(-torch.log(a) / self.spec.power)))

    def forward(self, x, batch: RaggedBatch, cache, mm: Callable):
        s = self.spec
        proj = mm(x, self.in_proj.weight, self.in_proj.bias)
        o = ops.rglru(proj, self.conv_w, self.conv_b, self.gates, self.gates_b, self.lam, cache[0], cache[1], batch.cu_q,
                      batch.seq_lens, batch.state_slots, batch.max_q, s.power, singles=batch.singles)
        return mm(o, self.o_proj.weight), self.residual_gate(proj)


class GatedMLP(Sublayer):
    """``forward(x, mm)`` of a feed-forward: (result, logits of its residual gate or None)."""

    def __init__(self, cfg: ModelConfig, spec: GluSpec, dtype, device):
        super().__init__(cfg, spec, 2 * spec.ff)
        self.gate_up_proj = self.first_matrix(cfg, False, dtype, device)
        self.down_proj = Linear(spec.ff, cfg.hidden_size, False, dtype, device)

    def forward(self, x, mm: Callable):
        s = self.spec
        gu = mm(x, self.gate_up_proj.weight, self.gate_up_proj.bias)
        if s.act == "silu":
            h = ops.silu_glu(gu, s.ff)
        else:
            h = ops.gelu_tanh_glu(gu, s.ff) if s.act == "gelu_tanh" else ops.clamped_glu(gu, s.ff, s.limit, s.alpha)
        return mm(h, self.down_proj.weight), self.residual_gate(gu)


class PlainMLP(Sublayer):
    """Two matrices with an activation between them."""

    def __init__(self, cfg: ModelConfig, spec: MlpSpec, dtype, device):
        super().__init__(cfg, spec, spec.ff)
        self.up_proj = self.first_matrix(cfg, False, dtype, device)
        self.down_proj = Linear(spec.ff, cfg.hidden_size, False, dtype, device)

    def forward(self, x, mm: Callable):
        u = mm(x, self.up_proj.weight, self.up_proj.bias)
        return mm(ops.activation(u, self.spec.ff, self.spec.act), self.down_proj.weight), self.residual_gate(u)


class RoutedMLP(Sublayer):
    """Mixture of experts; its result is still in parts (:class:`~verl_b200.ops.moe.RoutedSum`), which the next add + norm puts
    together. The residual gate goes with the shared unit's first matrix, or has one of its own."""

    def __init__(self, cfg: ModelConfig, spec: MoeSpec, dtype, device):
        super().__init__(cfg, spec, 0)
        H = cfg.hidden_size
        self.router_proj = Linear(H, pad8(spec.router_rows), False, dtype, device)  # router | gate of the shared unit
        first = torch.zeros(spec.experts, (2 if spec.gated else 1) * spec.ff, H, dtype=dtype, device=device)
        if spec.gated:
            self.experts_gate_up = nn.Parameter(first)
        else:
            self.experts_up = nn.Parameter(first)
        self.experts_down = nn.Parameter(torch.zeros(spec.experts, H, spec.ff, dtype=dtype, device=device))
        self.correction = (nn.Parameter(torch.zeros(spec.experts, dtype=torch.float32, device=device)) if spec.correction
                           else None)
        if spec.shared_ff:
            self.shared = (GatedMLP if spec.gated else PlainMLP)(cfg, spec.shared, dtype, device)
        elif self.gate_rows:
            self.gate_proj = self.first_matrix(cfg, False, dtype, device)
        # tokens per expert while a step is being routed; zero between steps
        self.register_buffer("counters", torch.zeros(spec.experts + 1, dtype=torch.int32, device=device), persistent=False)

    def reset_parameters(self, generator=None):
        with torch.no_grad():
            for w in (self.experts_first, self.experts_down):
                for e in range(w.shape[0]):
                    w[e].copy_(torch.empty(w.shape[1:], device=w.device).normal_(0.0, 0.02, generator=generator))

    @property
    def experts_first(self):
        return self.experts_gate_up if self.spec.gated else self.experts_up

    def forward(self, x, mm: Callable):
        s = self.spec
        logits = ops.gemm(x, self.router_proj.weight, out_dtype=torch.float32)
        routing = ops.moe_route(logits, s.experts, s.top, self.counters, score=s.score, renormalize=s.renormalize,
                                correction=self.correction)
        out = ops.moe_experts(x, routing, self.experts_first, self.experts_down, s.act, weigh_input=s.weigh == "input")
        shared = gate = None
        if s.shared_ff:
            shared, gate = self.shared(x, mm)
        elif self.gate_rows:
            gate = self.residual_gate(mm(x, self.gate_proj.weight, self.gate_proj.bias))
        return ops.RoutedSum(out, routing, s.weigh == "output", shared,
                             logits[:, s.experts] if s.shared_ff and s.shared_gate else None), gate


class SideInput(nn.Module):
    """Input of a layer's own per token: the layer's part of the token's side embedding, gated by the stream."""

    def __init__(self, cfg: ModelConfig, index: int, dtype, device):
        super().__init__()
        self.lo, self.dim = index * cfg.side_dim, cfg.side_dim
        self.gate_proj = Linear(cfg.hidden_size, cfg.side_dim, False, dtype, device)
        self.out_proj = Linear(cfg.side_dim, cfg.hidden_size, False, dtype, device)
        self.norm = RMSNormWeight(cfg.hidden_size, dtype, device)

    def forward(self, x, ids, table, mm: Callable):
        g = ops.gelu_rows(mm(x, self.gate_proj.weight), ids, table, self.lo, self.dim)
        return mm(g, self.out_proj.weight)


_MIXERS = {"attention": AttentionMixer, "latent_attention": LatentMixer, "delta": DeltaMixer, "gla": GlaMixer, "rglru": LruMixer}
_MLPS = {GluSpec: GatedMLP, MlpSpec: PlainMLP, MoeSpec: RoutedMLP}


def add_norm(pending, res, weight, eps, dtype):
    """Adds a sublayer's output (None: nothing) to the stream in place; the normed stream, or without a weight a copy."""
    if isinstance(pending, ops.RoutedSum):
        return ops.moe_combine(pending, res, weight, eps)
    return ops.add_rmsnorm(pending, res, weight, eps, dtype)


def norm_add(pending, gate, res, weight, eps, **after):
    """Adds the norm of a sublayer's output, times the sigmoid of ``gate`` where there is one, to the stream in place."""
    if isinstance(pending, ops.RoutedSum):
        return ops.moe_norm_add(pending, res, weight, eps, gate=gate, **after)
    return ops.rmsnorm_add(pending, res, weight, eps, gate=gate, **after)


class HybridLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: LayerSpec, index: int, dtype, device):
        super().__init__()
        both = cfg.design.norm == "both"  # norm1, norm2 in front of the sublayers, norm1b, norm2b behind them
        self.norm1 = RMSNormWeight(cfg.hidden_size, dtype, device)
        self.norm1b = RMSNormWeight(cfg.hidden_size, dtype, device) if both else None
        self.mixer = _MIXERS[spec.kind](cfg, spec.mixer, dtype, device)
        if spec.mlp is not None:
            self.norm2 = RMSNormWeight(cfg.hidden_size, dtype, device)
            self.norm2b = RMSNormWeight(cfg.hidden_size, dtype, device) if both else None
            self.mlp = _MLPS[type(spec.mlp)](cfg, spec.mlp, dtype, device)
        else:
            self.norm2 = self.norm2b = self.mlp = None
        self.side = SideInput(cfg, index, dtype, device) if cfg.side_dim else None


class HybridLM(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu"):
        super().__init__()
        self.cfg = cfg
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device)
        routed = any(isinstance(s.mlp, MoeSpec) for s in cfg.layer_specs)
        if cfg.design.norm == "post" and routed or cfg.design.norm != "pre" and cfg.side_dim:
            raise NotImplementedError("mixtures of experts and side inputs go with norms in front of the sublayers")
        if cfg.design.norm != "both" and cfg.design.residual_gate:
            raise NotImplementedError("residual gates go with norms on both sides of the sublayers")
        if cfg.has_position_table:
            self.pos_embed = nn.Embedding(cfg.max_position_embeddings, cfg.hidden_size, dtype=dtype, device=device)
        if cfg.design.embedding == "norm":
            self.embed_norm = RMSNormWeight(cfg.hidden_size, dtype, device)
        if cfg.side_dim:
            self.side_embed = nn.Embedding(cfg.vocab_size, cfg.num_hidden_layers * cfg.side_dim, dtype=dtype, device=device)
        # a layer that uses another's weights has no module of its own; ``runs`` has the module of every layer
        own = [weight_owner(cfg.layer_specs, i) for i in range(len(cfg.layer_specs))]
        self.layers = nn.ModuleList([HybridLayer(cfg, s, i, dtype, device) if own[i] == i else None
                                     for i, s in enumerate(cfg.layer_specs)])
        self.runs = tuple(self.layers[j] for j in own)
        self.norm = RMSNormWeight(cfg.hidden_size, dtype, device)
        self.lm_head = None if cfg.tie_word_embeddings else Linear(cfg.hidden_size, cfg.vocab_size, False, dtype, device)
        # portions up to this many tokens run latent attention in the latent space; sizes without an expanded form: all
        self.latent_short = LATENT_SHORT
        for s in cfg.layer_specs:
            m = s.mixer
            if s.kind == "latent_attention" and not ops.latent_prefill_supported(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank,
                                                                                 dtype, device):
                self.latent_short = 1 << 30

    def init_weights(self, seed: int = 0):
        dev = self.embed_tokens.weight.device
        gen = torch.Generator(device=dev)
        gen.manual_seed(seed)
        with torch.no_grad():
            for e in (self.embed_tokens, getattr(self, "side_embed", None), getattr(self, "pos_embed", None)):
                if e is not None:  # a table that is the output projection as well: logits of a size near one
                    std = self.cfg.hidden_size ** -0.5 if self.cfg.tie_word_embeddings and e is self.embed_tokens else 1.0
                    std = 0.3 if e is getattr(self, "pos_embed", None) else std
                    e.weight.copy_(torch.empty(e.weight.shape, dtype=torch.float32, device=dev).normal_(0.0, std, generator=gen))
        for m in self.modules():
            if isinstance(m, (Linear, DeltaMixer, GlaMixer, LruMixer, RoutedMLP)):
                m.reset_parameters(gen)
            elif isinstance(m, AttentionMixer) and m.spec.bias_rows:
                with torch.no_grad():
                    m.rel.copy_(torch.empty(m.rel.shape, device=dev).normal_(0.0, 0.5, generator=gen))
            if isinstance(m, (AttentionMixer, LatentMixer)) and m.spec.sink:
                with torch.no_grad():
                    m.sink.copy_(torch.empty(m.sink.shape, device=dev).normal_(0.0, 1.0, generator=gen))
            if isinstance(m, AttentionMixer):
                with torch.no_grad():  # distance biases of a few units; about one key in e^4 weighs one half
                    if m.spec.log_bias:
                        m.r1.uniform_(0.0, 1.0, generator=gen)
                        m.r2.uniform_(0.05, 0.5, generator=gen)
                    if m.spec.weighting == "sigmoid":
                        m.shift.fill_(-4.0)
        self.refresh()
        return self

    def refresh(self):
        """Derived tables, after the weights have changed."""
        for layer in self.layers:
            if layer is not None:
                layer.mixer.refresh()

    @property
    def lm_head_weight(self) -> torch.Tensor:
        return self.embed_tokens.weight if self.lm_head is None else self.lm_head.weight

    def projection_weights(self) -> list[torch.Tensor]:
        """Matrices of the layers (what weight quantisation applies to). Left out: the projections out of the latent, which are
        applied to queries and to weighted sums as well as to the latents; routers, whose scores choose; the narrow matrices of
        side inputs."""
        return [m.weight for layer in self.layers if layer is not None for n, m in layer.named_modules()
                if isinstance(m, Linear) and not n.endswith(("kv_up_proj", "router_proj")) and not n.startswith("side.")]

    def plan_latent(self, counts: list[int], ctx: list[int], boundaries: Callable) -> Optional[LatentPlan]:
        """How latent-attention layers run a step of ``counts[i]`` new tokens in sequences of ``ctx[i]`` tokens, ordered by
        :meth:`latent_order`. ``boundaries(list)``: int32 device tensor. None without such layers."""
        windows = {s.mixer.window for s in self.cfg.layer_specs if s.kind == "latent_attention"}
        if not windows:
            return None
        B = sum(c <= self.latent_short for c in counts)
        full = self._latent_groups(B, counts, ctx, boundaries) if 0 in windows else ()
        return LatentPlan(B, sum(counts[:B]), full,
                          {w: self._latent_groups(B, counts, [min(n, c + w - 1) for n, c in zip(ctx, counts)], boundaries)
                           for w in sorted(windows - {0})})

    @staticmethod
    def _latent_groups(B: int, counts: list[int], ctx: list[int], boundaries: Callable) -> tuple:
        groups, b0 = [], B
        while b0 < len(counts):  # expanded keys and values are scratch: contexts are taken together up to a bound
            b1, total = b0 + 1, ctx[b0]
            while b1 < len(counts) and total + ctx[b1] <= LATENT_GROUP:
                total += ctx[b1]
                b1 += 1
            cu = [0]
            for c in ctx[b0:b1]:
                cu.append(cu[-1] + c)
            groups.append((b0, b1, boundaries(cu), total, max(counts[b0:b1])))
            b0 = b1
        return tuple(groups)

    def latent_order(self, counts: list[int]) -> Optional[list[int]]:
        """Order of a step's sequences: those whose latent attention stays in the latent space first, and where recurrent units
        step single tokens together, those before all others. None: any order."""
        kinds = {s.kind for s in self.cfg.layer_specs}
        if not kinds & {"latent_attention", "gla", "rglru"}:
            return None
        singles = bool(kinds & {"gla", "rglru"})
        return sorted(range(len(counts)), key=lambda i: (counts[i] > self.latent_short, singles and counts[i] > 1))

    def forward(self, *args, **kwargs):
        raise NotImplementedError(f"{self.cfg.model_type}: layer-list models are served by the rollout engine only "
                                  "(no training forward)")

    @torch.no_grad()
    def run(self, ids: torch.Tensor, batch: RaggedBatch, cache: StateCache, mm: Callable,
            observe: Optional[Callable] = None) -> torch.Tensor:
        """Final-norm hidden states [T, H] of one step (times the design's logit scale). ``mm(x, w)`` or ``mm(x, w, bias)``: the
        engine's matrix product. ``observe(i, stream)`` gets the residual stream after layer i (a copy; debugging and tests)."""
        c, eps, dtype = self.cfg, self.cfg.rms_norm_eps, self.embed_tokens.weight.dtype
        if c.design.norm == "post":
            res, x = ops.embedding_scaled(ids, self.embed_tokens.weight, c.embedding_scale, with_copy=True)
            last = len(self.layers) - 1
            for i, layer in enumerate(self.runs):
                subs = [(lambda v: layer.mixer(v, batch, cache.layers[i], mm)[0], layer.norm1)]
                if layer.mlp is not None:
                    subs.append((lambda v: layer.mlp(v, mm)[0], layer.norm2))
                for k, (sub, norm) in enumerate(subs):
                    final = self.norm.weight if i == last and k == len(subs) - 1 else None
                    x = ops.rmsnorm_add(sub(x), res, norm.weight, eps, final_weight=final, final_scale=c.logit_scale)
                if observe is not None:
                    observe(i, res.clone())
            return x
        if c.design.embedding == "norm":
            res = ops.embedding_normed(ids, self.embed_tokens.weight, self.embed_norm.weight, eps)
        elif c.design.embedding == "positions":
            res = ops.embedding_scaled(ids, self.embed_tokens.weight, c.embedding_scale, pos_table=self.pos_embed.weight,
                                       positions=batch.positions)
        else:
            res = ops.embedding_scaled(ids, self.embed_tokens.weight, c.embedding_scale)
        x = ops.add_rmsnorm(None, res, self.runs[0].norm1.weight, eps)
        last = len(self.runs) - 1
        for i, layer in enumerate(self.runs):
            # the norm that the next sublayer (or the head) reads through
            after = (self.runs[i + 1].norm1 if i < last else self.norm).weight
            pending, gate = layer.mixer(x, batch, cache.layers[i], mm)
            if c.design.norm == "both":
                end = {"final_weight": after, "final_scale": c.logit_scale if i == last else 1.0}
                if layer.mlp is not None:
                    x = norm_add(pending, gate, res, layer.norm1b.weight, eps, final_weight=layer.norm2.weight)
                    x = norm_add(*layer.mlp(x, mm), res, layer.norm2b.weight, eps, **end)
                else:
                    x = norm_add(pending, gate, res, layer.norm1b.weight, eps, **end)
                if observe is not None:
                    observe(i, res.clone())
                continue
            if layer.mlp is not None:
                x = add_norm(pending, res, layer.norm2.weight, eps, dtype)
                pending, _ = layer.mlp(x, mm)
            if layer.side is not None:
                y = layer.side(add_norm(pending, res, None, eps, dtype), ids, self.side_embed.weight, mm)
                x = ops.rmsnorm_add(y, res, layer.side.norm.weight, eps, final_weight=after)
            else:
                x = add_norm(pending, res, after, eps, dtype)
            if observe is not None:
                observe(i, res.clone())
        return x
