"""Decoders described layer by layer (``ModelConfig.layer_specs``): every layer has its own mixer, softmax attention over
the paged KV cache or a gated delta rule with per-sequence state, and an optional clamped-GLU feed-forward.

Served by the rollout engine like the homogeneous stacks of :mod:`.transformer`; there is no training path. The residual
stream is fp32 and every norm is fused with the residual add in front of it:

    embedding * scale -> [ add + norm1 -> fused input projection -> mixer -> output projection
                           -> add + norm2 -> gate|up -> clamped GLU -> down ] ... -> add + final norm -> head
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Optional

import torch
import torch.nn as nn

from .. import ops
from .config import ModelConfig
from .layer_specs import AttentionSpec, DeltaSpec, GluSpec, LayerSpec, distance_buckets
from .transformer import Linear, RMSNormWeight


def pad8(n: int) -> int:
    """Rows of a fused projection: a multiple of 8 keeps the rows of its output 16-byte aligned."""
    return (n + 7) // 8 * 8


@dataclass
class RaggedBatch:
    """One step: the new tokens of B sequences, described for the cache and state (all int32 except ``slots`` int64)."""

    cu_q: torch.Tensor         # [B + 1] boundaries of the new tokens
    max_q: int
    seq_lens: torch.Tensor     # [B] tokens of each sequence including the new ones
    slots: torch.Tensor        # [T] cache place of each token (page * block_size + offset; < 0: padding)
    block_table: torch.Tensor  # [B, max_blocks]
    state_slots: torch.Tensor  # [B] recurrent-state slot (< 0: padding)
    max_ctx: int = 0           # longest sequence a replay of this step may see
    work: dict = field(default_factory=dict)  # scratch owned by the caller (CUDA graphs)


class StateCache:
    """Cache of a layer-list model: K / V pages per attention layer, fp32 state and convolution ring per delta layer."""

    def __init__(self, cfg: ModelConfig, num_blocks: int, block_size: int, num_slots: int, dtype, device):
        self.layers: list[tuple] = []
        for spec in cfg.layer_specs:
            m = spec.mixer
            if spec.kind == "attention":
                self.layers.append(tuple(torch.zeros((num_blocks, m.kv_heads, block_size, d), dtype=dtype, device=device)
                                         for d in (m.dim, m.vdim)))
            else:
                self.layers.append((torch.zeros((num_slots, m.conv, m.channels), dtype=dtype, device=device),
                                    torch.zeros((num_slots, m.heads, m.vdim, m.dim), dtype=torch.float32, device=device)))

    @staticmethod
    def page_bytes(cfg: ModelConfig, block_size: int, itemsize: int) -> int:
        return sum(s.mixer.kv_heads * (s.mixer.dim + s.mixer.vdim) for s in cfg.layer_specs
                   if s.kind == "attention") * block_size * itemsize

    @staticmethod
    def slot_bytes(cfg: ModelConfig, itemsize: int) -> int:
        return sum(m.conv * m.channels * itemsize + 4 * m.heads * m.vdim * m.dim
                   for m in (s.mixer for s in cfg.layer_specs if s.kind == "delta"))


class AttentionMixer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: AttentionSpec, dtype, device):
        super().__init__()
        self.spec, self.eps = spec, cfg.rms_norm_eps
        self.qkv_proj = Linear(cfg.hidden_size, pad8(spec.q_size + spec.k_size + spec.v_size), False, dtype, device)
        self.o_proj = Linear(spec.out_size, cfg.hidden_size, False, dtype, device)
        if spec.qk_norm:
            self.q_norm = RMSNormWeight(spec.q_size, dtype, device)
            self.k_norm = RMSNormWeight(spec.k_size, dtype, device)
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
        qkv = mm(x, self.qkv_proj.weight)
        q = ops.qk_norm_kv_write(qkv, *norms, batch.slots, cache[0], cache[1], s.heads, self.eps)
        o = ops.paged_attention(q, cache[0], cache[1], batch.block_table, batch.cu_q, batch.seq_lens, batch.max_q,
                                scale=s.scale, window=s.window, keep_first=s.keep_first,
                                bias=self.bias if s.bias_rows else None, max_ctx=batch.max_ctx)
        return mm(o, self.o_proj.weight)


class DeltaMixer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: DeltaSpec, dtype, device):
        super().__init__()
        self.spec, self.eps = spec, cfg.rms_norm_eps
        self.in_proj = Linear(cfg.hidden_size, pad8(spec.proj_size), False, dtype, device)
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

    def refresh(self):
        pass

    def forward(self, x, batch: RaggedBatch, cache, mm: Callable):
        s = self.spec
        proj = mm(x, self.in_proj.weight)
        o = ops.delta_rule(proj, self.conv, self.A_log, self.dt_bias, self.norm.weight, cache[0], cache[1], batch.cu_q,
                           batch.seq_lens, batch.state_slots, batch.max_q, s.heads, s.kv_heads, s.dim, s.vdim, self.eps)
        return mm(o, self.o_proj.weight)


class ClampedGLU(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: GluSpec, dtype, device):
        super().__init__()
        self.spec = spec
        self.gate_up_proj = Linear(cfg.hidden_size, pad8(2 * spec.ff), False, dtype, device)
        self.down_proj = Linear(spec.ff, cfg.hidden_size, False, dtype, device)

    def forward(self, x, mm: Callable):
        s = self.spec
        return mm(ops.clamped_glu(mm(x, self.gate_up_proj.weight), s.ff, s.limit, s.alpha), self.down_proj.weight)


class HybridLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: LayerSpec, dtype, device):
        super().__init__()
        self.norm1 = RMSNormWeight(cfg.hidden_size, dtype, device)
        mixer = AttentionMixer if spec.kind == "attention" else DeltaMixer
        self.mixer = mixer(cfg, spec.mixer, dtype, device)
        if spec.mlp is not None:
            self.norm2 = RMSNormWeight(cfg.hidden_size, dtype, device)
            self.mlp = ClampedGLU(cfg, spec.mlp, dtype, device)
        else:
            self.norm2 = self.mlp = None


class HybridLM(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu"):
        super().__init__()
        self.cfg = cfg
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device)
        self.layers = nn.ModuleList([HybridLayer(cfg, s, dtype, device) for s in cfg.layer_specs])
        self.norm = RMSNormWeight(cfg.hidden_size, dtype, device)
        self.lm_head = Linear(cfg.hidden_size, cfg.vocab_size, False, dtype, device)

    def init_weights(self, seed: int = 0):
        dev = self.embed_tokens.weight.device
        gen = torch.Generator(device=dev)
        gen.manual_seed(seed)
        with torch.no_grad():
            w = self.embed_tokens.weight
            w.copy_(torch.empty(w.shape, dtype=torch.float32, device=dev).normal_(0.0, 1.0, generator=gen))
        for m in self.modules():
            if isinstance(m, (Linear, DeltaMixer)):
                m.reset_parameters(gen)
            elif isinstance(m, AttentionMixer) and m.spec.bias_rows:
                with torch.no_grad():
                    m.rel.copy_(torch.empty(m.rel.shape, device=dev).normal_(0.0, 0.5, generator=gen))
        self.refresh()
        return self

    def refresh(self):
        """Derived tables, after the weights have changed."""
        for layer in self.layers:
            layer.mixer.refresh()

    @property
    def lm_head_weight(self) -> torch.Tensor:
        return self.lm_head.weight

    def projection_weights(self) -> list[torch.Tensor]:
        """Matrices of the layers (what weight quantisation applies to)."""
        return [m.weight for layer in self.layers for m in layer.modules() if isinstance(m, Linear)]

    def forward(self, *args, **kwargs):
        raise NotImplementedError(f"{self.cfg.model_type}: layer-list models are served by the rollout engine only "
                                  "(no training forward)")

    @torch.no_grad()
    def run(self, ids: torch.Tensor, batch: RaggedBatch, cache: StateCache, mm: Callable,
            observe: Optional[Callable] = None) -> torch.Tensor:
        """Final-norm hidden states [T, H] of one step. ``mm(x, w)``: the engine's matrix product. ``observe(i, stream)``
        gets the residual stream after layer i (a copy; debugging and tests)."""
        eps = self.cfg.rms_norm_eps
        res = ops.embedding_scaled(ids, self.embed_tokens.weight, self.cfg.embedding_scale)
        pending = None  # output of the last sublayer, not yet added to the stream
        for i, layer in enumerate(self.layers):
            x = ops.add_rmsnorm(pending, res, layer.norm1.weight, eps)
            pending = layer.mixer(x, batch, cache.layers[i], mm)
            if layer.mlp is not None:
                x = ops.add_rmsnorm(pending, res, layer.norm2.weight, eps)
                pending = layer.mlp(x, mm)
            if observe is not None:
                observe(i, res + pending.float())
        return ops.add_rmsnorm(pending, res, self.norm.weight, eps)
