"""Native ops of the framework. CUDA tensors run on the hand-written sm_100a kernels in
``verl_b200/csrc`` (loaded through :mod:`verl_b200.ops._lib`); CPU tensors take plain-torch
reference paths that exist for the CPU test tier."""

from . import _lib
from .attention import (attention_varlen, decode_workspace, head_norm_rope_kv_write, kv_cache_write, paged_attention,
                        paged_decode_attention, qk_norm_kv_write)
from .delta import delta_rule
from .gemm import gemm, linear
from .gla import gated_linear_attention
from .latent import (latent_attention, latent_gather, latent_prefill, latent_prefill_supported, latent_queries,
                     latent_rope_write, latent_values, latent_width, rotate_tails)
from .lmhead import lmhead_logprob_entropy
from .lru import rglru
from .moe import RoutedSum, moe_combine, moe_experts, moe_norm_add, moe_route
from .nn import (activation, add_rmsnorm, clamped_glu, embedding, embedding_normed, embedding_scaled, gelu_rows, gelu_tanh_glu,
                 rmsnorm, rmsnorm_add, rope_qkv, rope_tables, silu_glu, softcap_, swiglu)
from .rl import (PPO_METRIC_NAMES, adamw_step, clip_coef, decode_advance, gae, grpo_advantage, ppo_loss_fused, sample,
                 sumsq_into)

__all__ = [
    "_lib", "gemm", "linear", "lmhead_logprob_entropy", "embedding", "rmsnorm", "rope_qkv", "rope_tables", "swiglu",
    "attention_varlen", "paged_decode_attention", "kv_cache_write", "decode_workspace", "ppo_loss_fused", "gae",
    "grpo_advantage", "sample", "decode_advance", "adamw_step", "sumsq_into", "clip_coef", "PPO_METRIC_NAMES",
    "paged_attention", "qk_norm_kv_write", "delta_rule", "add_rmsnorm", "clamped_glu", "embedding_scaled",
    "rmsnorm_add", "gelu_tanh_glu", "head_norm_rope_kv_write", "latent_attention", "latent_gather", "latent_prefill",
    "latent_prefill_supported", "latent_queries", "latent_rope_write", "latent_values", "latent_width", "rotate_tails",
    "embedding_normed", "silu_glu", "gelu_rows", "softcap_", "rglru", "RoutedSum", "moe_route", "moe_experts", "moe_combine",
    "activation", "gated_linear_attention", "moe_norm_add",
]
