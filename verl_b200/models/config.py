"""Architecture description shared by the training engine, the rollout engine and the
checkpoint code. Mirrors the HF ``config.json`` fields of the supported families
(Llama, Qwen2/2.5, Qwen3, Qwen3-MoE); the reference gets these models from
``transformers`` (verl/utils/model.py:103-127)."""

from __future__ import annotations

import json
from dataclasses import asdict, dataclass, field, replace
from pathlib import Path
from typing import Any

from .layer_specs import (DESIGNS, AttentionSpec, DeltaSpec, Design, GlaSpec, GluSpec, LatentSpec, LayerSpec, LruSpec, MlpSpec,
                          MoeSpec, RotarySpec, weight_owner)

_ARCH_TO_TYPE = {
    "LlamaForCausalLM": "llama",
    "MistralForCausalLM": "llama",
    "Qwen2ForCausalLM": "qwen2",
    "Qwen3ForCausalLM": "qwen3",
    "Qwen3MoeForCausalLM": "qwen3_moe",
    "ApertusForCausalLM": "apertus",
    "Qwen2VLForConditionalGeneration": "qwen2_vl",
    "Qwen2_5_VLForConditionalGeneration": "qwen2_5_vl",
    "Qwen3VLForConditionalGeneration": "qwen3_vl",
    "Qwen3VLMoeForConditionalGeneration": "qwen3_vl_moe",
    "LlamaForTokenClassification": "llama",
    "Qwen2ForTokenClassification": "qwen2",
    "Qwen3ForTokenClassification": "qwen3",
}
_TYPE_TO_ARCH = {"llama": "LlamaForCausalLM", "qwen2": "Qwen2ForCausalLM", "qwen3": "Qwen3ForCausalLM",
                 "qwen3_moe": "Qwen3MoeForCausalLM", "qwen2_vl": "Qwen2VLForConditionalGeneration",
                 "qwen2_5_vl": "Qwen2_5_VLForConditionalGeneration", "apertus": "ApertusForCausalLM",
                 "qwen3_vl": "Qwen3VLForConditionalGeneration", "qwen3_vl_moe": "Qwen3VLMoeForConditionalGeneration"}
# designs whose config.json lists its layers one by one (``architecture`` instead of ``architectures``)
_LAYER_LIST_ARCHS = {"Fuganex": "fuganex", "Padodra": "padodra", "Golonex": "golonex", "Malinex": "malinex"}
_VL_TYPES = ("qwen2_vl", "qwen2_5_vl", "qwen3_vl", "qwen3_vl_moe")


@dataclass
class ModelConfig:
    model_type: str = "qwen2"
    vocab_size: int = 152064
    hidden_size: int = 3584
    intermediate_size: int = 18944
    num_hidden_layers: int = 28
    num_attention_heads: int = 28
    num_key_value_heads: int = 4
    head_dim: int | None = None
    rope_theta: float = 1e6
    rms_norm_eps: float = 1e-6
    max_position_embeddings: int = 32768
    tie_word_embeddings: bool = False
    attention_bias: bool | None = None  # None -> family default (qwen2: True)
    qk_norm: bool | None = None  # None -> family default (qwen3*, apertus: True)
    # "silu": gated SwiGLU MLP (gate / up / down); "xielu": Apertus' two-matrix MLP with the learnable xIELU activation
    hidden_act: str | None = None
    # MoE (qwen3_moe)
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    router_aux_loss_coef: float = 0.0
    # token-classification / value head
    num_labels: int = 0
    bos_token_id: int | None = None
    eos_token_id: int | None = 2
    pad_token_id: int | None = None
    # layer-list designs: one LayerSpec per layer (empty: all layers alike, described by the fields above)
    layer_specs: tuple = ()
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    logit_softcap: float = 0.0  # > 0: logits become softcap * tanh(logits / softcap)
    side_dim: int = 0           # size of the per-token input of every layer (0 = none)
    extra: dict = field(default_factory=dict)

    def __post_init__(self):
        self.layer_specs = tuple(self.layer_specs)
        if self.layer_specs:
            self.num_hidden_layers = len(self.layer_specs)
            for i in range(len(self.layer_specs)):
                weight_owner(self.layer_specs, i)
            self.tie_word_embeddings = self.design.tied
        if self.head_dim is None:
            self.head_dim = self.hidden_size // self.num_attention_heads
        if self.attention_bias is None:
            self.attention_bias = self.model_type in ("qwen2", "qwen2_vl", "qwen2_5_vl")
        if self.qk_norm is None:
            self.qk_norm = self.model_type in ("qwen3", "qwen3_moe", "apertus", "qwen3_vl", "qwen3_vl_moe")
        if self.hidden_act is None:
            self.hidden_act = "xielu" if self.model_type == "apertus" else "silu"

    # ------------------------------------------------------------------ derived
    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_layer_list(self) -> bool:
        return bool(self.layer_specs)

    @property
    def design(self) -> Design:
        """What the layer-list design fixes for all its models."""
        return DESIGNS[self.model_type]

    @property
    def has_recurrent_state(self) -> bool:
        """Some layer carries a state per sequence that pages cannot share."""
        return any(s.kind in ("delta", "gla", "rglru") for s in self.layer_specs)

    @property
    def has_position_table(self) -> bool:
        """Positions are rows of a learned table: no sequence is longer than ``max_position_embeddings``."""
        return self.is_layer_list and self.design.embedding == "positions"

    @property
    def mlp_gated(self) -> bool:
        return self.hidden_act != "xielu"

    # vision-language models (Qwen2-VL family): the decoder fields above describe the language model; the vision tower,
    # the placeholder token ids and the multimodal RoPE sections live in ``extra``
    @property
    def is_vl(self) -> bool:
        return bool(self.extra.get("vision_config"))

    @property
    def mrope_section(self):
        return self.extra.get("mrope_section")

    @property
    def mrope_interleaved(self) -> bool:
        """Qwen3-VL: the frequencies of the three axes alternate (T H W T H W ... T T) instead of lying in three
        consecutive sections."""
        return bool(self.extra.get("mrope_interleaved", False))

    @property
    def image_token_id(self) -> int:
        return int(self.extra.get("image_token_id", 151655))

    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_key_value_heads * self.head_dim

    def num_parameters(self, include_embedding: bool = True) -> int:
        H, L = self.hidden_size, self.num_hidden_layers
        if self.is_layer_list:
            total = H + sum(s.num_parameters(H, self.design) for s in self.layer_specs)
            if self.has_position_table and include_embedding:
                total += self.max_position_embeddings * H
            if self.design.embedding == "norm":
                total += H
            if self.side_dim:
                total += L * (2 * H * self.side_dim + H)
                if include_embedding:
                    total += self.vocab_size * L * self.side_dim
            return total + ((1 if self.tie_word_embeddings else 2) * self.vocab_size * H if include_embedding else 0)
        attn = H * (self.q_size + 2 * self.kv_size) + self.q_size * H
        if self.attention_bias:
            attn += self.q_size + 2 * self.kv_size
        if self.qk_norm:
            attn += 2 * self.head_dim
        if self.is_moe:
            mlp = self.num_experts * 3 * H * self.moe_intermediate_size + H * self.num_experts
        else:
            mlp = (3 if self.mlp_gated else 2) * H * self.intermediate_size + (0 if self.mlp_gated else 2)
        total = L * (attn + mlp + 2 * H) + H
        if include_embedding:
            total += self.vocab_size * H * (1 if self.tie_word_embeddings else 2)
        return total

    # --------------------------------------------------------------- (de)serialise
    @classmethod
    def from_hf_dict(cls, d: dict[str, Any]) -> "ModelConfig":
        if d.get("architecture") in _LAYER_LIST_ARCHS:
            return cls._from_layer_list(d)
        mt = d.get("model_type")
        if mt is None:
            archs = d.get("architectures") or ["Qwen2ForCausalLM"]
            mt = _ARCH_TO_TYPE.get(archs[0], "qwen2")
        if mt in _VL_TYPES:  # language-model fields are nested under text_config in recent HF versions
            top = {k: v for k, v in d.items() if k not in ("text_config", "vision_config")}
            flat = dict(top)
            flat.update(d.get("text_config") or {})
            rope = flat.get("rope_scaling") or flat.get("rope_parameters") or {}
            flat["model_type"] = mt
            extra_vl = {"vision_config": dict(d.get("vision_config") or {}),
                        "mrope_section": list(rope.get("mrope_section") or []) or None}
            if rope.get("mrope_interleaved") or mt in ("qwen3_vl", "qwen3_vl_moe"):
                extra_vl["mrope_interleaved"] = True
            if "rope_theta" not in flat and rope.get("rope_theta"):
                flat["rope_theta"] = rope["rope_theta"]
            for k in ("image_token_id", "video_token_id", "vision_start_token_id", "vision_end_token_id"):
                if k in top:
                    extra_vl[k] = top[k]
            d = {k: v for k, v in flat.items() if k not in ("rope_scaling", "rope_parameters", "image_token_id",
                                                            "video_token_id", "vision_start_token_id", "vision_end_token_id")}
            d["_vl_extra"] = extra_vl
        else:
            # text models: recent HF versions nest theta and the scaling rule under rope_parameters
            rope = d.get("rope_parameters") or d.get("rope_scaling") or None
            if isinstance(rope, dict):
                d = dict(d)
                if d.get("rope_theta") is None and rope.get("rope_theta") is not None:
                    d["rope_theta"] = rope["rope_theta"]
                kind = rope.get("rope_type") or rope.get("type") or "default"
                d.pop("rope_parameters", None)
                d.pop("rope_scaling", None)
                if kind != "default":
                    d["rope_scaling"] = {k: v for k, v in rope.items() if k != "rope_theta"}
        known = {f for f in cls.__dataclass_fields__}
        may_be_none = ("eos_token_id", "pad_token_id", "bos_token_id", "head_dim", "attention_bias", "qk_norm", "hidden_act")
        kw = {k: v for k, v in d.items() if k in known and k != "extra" and (v is not None or k in may_be_none)}
        kw["model_type"] = mt
        if "num_local_experts" in d and "num_experts" not in d:
            kw["num_experts"] = d["num_local_experts"]
        eos = kw.get("eos_token_id")
        if isinstance(eos, list):
            kw["eos_token_id"] = eos[0]
        cfg = cls(**kw)
        if cfg.is_moe and (d.get("mlp_only_layers") or int(d.get("decoder_sparse_step") or 1) != 1):
            raise NotImplementedError("mixture-of-experts stacks with dense layers in between (mlp_only_layers, "
                                      "decoder_sparse_step != 1) are not supported: every layer is sparse here")
        cfg.extra = {k: v for k, v in d.items() if k not in known and k != "_vl_extra"}
        cfg.extra.update(d.get("_vl_extra") or {})
        return cfg

    @classmethod
    def _from_layer_list(cls, d: dict[str, Any]) -> "ModelConfig":
        model_type = _LAYER_LIST_ARCHS[d["architecture"]]
        design = DESIGNS[model_type]
        specs = tuple(LayerSpec.from_dict(x, design) for x in d["layers"])
        att = [s.mixer for s in specs if s.kind == "attention"]
        kw = {k: int(d[k]) for k in ("bos_token_id", "eos_token_id", "pad_token_id") if d.get(k) is not None}
        kw.setdefault("eos_token_id", None)
        known = ["architecture", "vocab", "width", "layers", "norm", *kw]
        if design.embedding == "scale":
            known.append("embedding")
            kw["embedding_scale"] = float(d["embedding"]["scale"])
        elif design.embedding == "positions":
            known.append("max_positions")
            if d.get("max_positions") is not None:
                kw["max_position_embeddings"] = int(d["max_positions"])
        if design.logit_scale:
            known.append("logit_scale")
            kw["logit_scale"] = float(d.get("logit_scale", 1.0))
        if design.logit_softcap:
            known.append("logit_softcap")
            kw["logit_softcap"] = float(d.get("logit_softcap") or 0.0)
        if design.side:
            known.append("token_side")
            kw["side_dim"] = int((d.get("token_side") or {}).get("dim") or 0)
        return cls(model_type=model_type, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                   intermediate_size=max([s.mlp.ff for s in specs if s.mlp] or [0]),
                   num_attention_heads=max([a.heads for a in att] or [1]),
                   num_key_value_heads=max([a.kv_heads for a in att] or [1]), head_dim=max([a.dim for a in att] or [1]),
                   rms_norm_eps=float(d["norm"]["eps"]),
                   layer_specs=specs, extra={k: v for k, v in d.items() if k not in known}, **kw)

    def _to_layer_list(self) -> dict[str, Any]:
        arch = {v: k for k, v in _LAYER_LIST_ARCHS.items()}[self.model_type]
        d = {"architecture": arch, "vocab": self.vocab_size, "width": self.hidden_size,
             "layers": [s.to_dict() for s in self.layer_specs], "norm": {"eps": self.rms_norm_eps}, **self.extra}
        if self.design.embedding == "scale":
            d["embedding"] = {"scale": self.embedding_scale}
        elif self.has_position_table:
            d["max_positions"] = self.max_position_embeddings
        if self.design.logit_scale:
            d["logit_scale"] = self.logit_scale
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        if self.side_dim:
            d["token_side"] = {"dim": self.side_dim}
        for k in ("bos_token_id", "eos_token_id", "pad_token_id"):
            if getattr(self, k) is not None:
                d[k] = getattr(self, k)
        return d

    @classmethod
    def from_pretrained(cls, path: str | Path) -> "ModelConfig":
        p = Path(path)
        if p.is_dir():
            p = p / "config.json"
        return cls.from_hf_dict(json.loads(p.read_text()))

    def to_hf_dict(self) -> dict[str, Any]:
        if self.is_layer_list:
            return self._to_layer_list()
        d = asdict(self)
        for k in ("layer_specs", "embedding_scale", "logit_scale", "logit_softcap", "side_dim"):
            del d[k]
        extra = d.pop("extra")
        if self.model_type in _VL_TYPES:
            moe_keys = () if self.is_moe else ("num_experts", "num_experts_per_tok", "moe_intermediate_size", "norm_topk_prob",
                                               "router_aux_loss_coef")
            text = {k: v for k, v in d.items() if k not in moe_keys + ("num_labels",)}
            text["model_type"] = self.model_type + "_text"
            text["rope_scaling"] = {"type": "mrope", "mrope_section": list(extra.get("mrope_section") or [])}
            if self.model_type in ("qwen3_vl", "qwen3_vl_moe"):
                text["rope_scaling"] = {"rope_type": "default", "mrope_section": list(extra.get("mrope_section") or []),
                                        "mrope_interleaved": True, "rope_theta": self.rope_theta}
            out = {"architectures": [_TYPE_TO_ARCH[self.model_type]], "model_type": self.model_type, "torch_dtype": "bfloat16",
                   "text_config": text, "vision_config": dict(extra.get("vision_config") or {}),
                   "tie_word_embeddings": self.tie_word_embeddings}
            for k in ("image_token_id", "video_token_id", "vision_start_token_id", "vision_end_token_id"):
                if k in extra:
                    out[k] = extra[k]
            return out
        arch = _TYPE_TO_ARCH.get(self.model_type, "Qwen2ForCausalLM")
        if self.num_labels:
            arch = arch.replace("ForCausalLM", "ForTokenClassification")
        d["architectures"] = [arch]
        d["torch_dtype"] = "bfloat16"
        if not self.is_moe:
            for k in ("num_experts", "num_experts_per_tok", "moe_intermediate_size", "norm_topk_prob",
                      "router_aux_loss_coef"):
                d.pop(k)
        if not self.num_labels:
            d.pop("num_labels")
        d.update({k: v for k, v in extra.items() if k not in d})
        return d

    def save_pretrained(self, path: str | Path) -> None:
        p = Path(path)
        p.mkdir(parents=True, exist_ok=True)
        (p / "config.json").write_text(json.dumps(self.to_hf_dict(), indent=2))


def _fuganex_specs(groups: int, heads: int, kv_heads: int, dim: int, window: int, keep_first: int, ff: int, d_heads: int,
                   d_kv_heads: int, d_dim: int) -> tuple:
    """``groups`` x (two delta-rule layers, one attention layer), a feed-forward after each."""
    mlp = GluSpec(ff, 7.0)
    delta = LayerSpec(DeltaSpec(d_heads, d_kv_heads, d_dim, d_dim, 4), mlp)
    att = LayerSpec(AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window, keep_first, 128.0, 32), mlp)
    return (delta, delta, att) * groups


def _padodra_specs(groups: int, heads: int, kv_heads: int, dim: int, chunk: int, ff: int, latent: tuple) -> tuple:
    """``groups`` x (two chunked attention layers, one latent attention layer), a feed-forward after each. ``latent``: heads,
    unrotated and rotated head size, value size, rank."""
    mlp = GluSpec(ff, act="gelu_tanh")
    rot = RotarySpec(dim, 500000.0, True, (("factor", 8.0), ("high", 4.0), ("low", 1.0), ("original", 8192)))
    att = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, qk_norm="head", rotary=rot, chunk=chunk, softcap=30.0,
                        sink=True, gate="element")
    h, d, r, v, rank = latent
    yarn = RotarySpec(r, 10000.0, False, (("factor", 40.0), ("fast", 32.0), ("original", 4096), ("slow", 1.0)))
    lat = LatentSpec(h, d, r, v, rank, (d + r) ** -0.5, yarn, "element")
    return (LayerSpec(att, mlp), LayerSpec(att, mlp), LayerSpec(lat, mlp)) * groups


def _golonex_specs(groups: int, heads: int, kv_heads: int, dim: int, window: int, lru: tuple, latent: tuple, moe: tuple) -> tuple:
    """``groups`` x (recurrent block, latent attention, attention), a mixture of experts after each. ``lru``: width, blocks,
    taps; ``latent``: heads, unrotated and rotated head size, value size, rank, rank of the queries; ``moe``: experts, experts
    per token, their size, the shared unit's size."""
    mlp = MoeSpec(*moe)
    yarn = RotarySpec(dim // 2, 10000.0, True, (("factor", 8.0), ("fast", 32.0), ("original", 4096), ("slow", 1.0)))
    att = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window, qk_norm=None, rotary=yarn, key_values=True)
    h, d, r, v, rank, q_rank = latent
    lat = LatentSpec(h, d, r, v, rank, (d + r) ** -0.5, RotarySpec(r, 10000.0, True), "head", q_rank, window, True)
    return (LayerSpec(LruSpec(*lru), mlp), LayerSpec(lat, mlp), LayerSpec(att, mlp)) * groups


def _malinex_specs(groups: int, heads: int, kv_heads: int, dim: int, gla: tuple, ff: int, moe: tuple) -> tuple:
    """``groups`` x (two layers of gated linear attention, one attention layer), a mixture of experts after each but the first, which
    has a dense feed-forward; every second group uses the linear layers of the group before it again. ``gla``: heads, key and
    value size, tau, rank; ``moe``: experts, experts per token, their size, the shared unit's size."""
    mlp = MoeSpec(*moe, act="relu2", score="softmax", renormalize=True, weigh="output", gated=False, correction=True,
                  shared_gate=False)
    lin = LayerSpec(GlaSpec(*gla), mlp)
    att = LayerSpec(AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, gate="head", qkv_bias=True, q_temp=(0.1, 1024.0),
                                  log_bias=True, weighting="sigmoid"), mlp)
    out = []
    for g in range(groups):
        for k in (0, 1):
            again = g % 2 and 3 * (g - 1) + k > 0
            out.append(replace(lin, weights_of=3 * (g - 1) + k) if again else replace(lin, mlp=MlpSpec(ff)) if g + k == 0 else lin)
        out.append(att)
    return tuple(out)


# Named architectures used by the benchmarks and tests (random-init, no download needed).
PRESETS: dict[str, dict] = {
    "tiny-qwen2": dict(model_type="qwen2", vocab_size=2048, hidden_size=256, intermediate_size=688,
                       num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, rope_theta=1e6,
                       tie_word_embeddings=True, eos_token_id=2),
    "qwen2.5-0.5b": dict(model_type="qwen2", vocab_size=151936, hidden_size=896, intermediate_size=4864,
                         num_hidden_layers=24, num_attention_heads=14, num_key_value_heads=2, rope_theta=1e6,
                         tie_word_embeddings=True, eos_token_id=151645),
    "qwen2.5-7b": dict(model_type="qwen2", vocab_size=152064, hidden_size=3584, intermediate_size=18944,
                       num_hidden_layers=28, num_attention_heads=28, num_key_value_heads=4, rope_theta=1e6,
                       eos_token_id=151645),
    "qwen2.5-32b": dict(model_type="qwen2", vocab_size=152064, hidden_size=5120, intermediate_size=27648,
                        num_hidden_layers=64, num_attention_heads=40, num_key_value_heads=8, rope_theta=1e6,
                        eos_token_id=151645),
    "qwen3-30b-a3b": dict(model_type="qwen3_moe", vocab_size=151936, hidden_size=2048, intermediate_size=6144,
                          num_hidden_layers=48, num_attention_heads=32, num_key_value_heads=4, head_dim=128,
                          rope_theta=1e6, num_experts=128, num_experts_per_tok=8, moe_intermediate_size=768,
                          eos_token_id=151645),
    "tiny-qwen3-moe": dict(model_type="qwen3_moe", vocab_size=2048, hidden_size=256, intermediate_size=512,
                           num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, head_dim=64,
                           num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128, eos_token_id=2),
    "tiny-qwen2-vl": dict(model_type="qwen2_vl", vocab_size=2048, hidden_size=256, intermediate_size=512,
                          num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, rope_theta=1e6, eos_token_id=2,
                          extra={"vision_config": dict(depth=2, embed_dim=64, hidden_size=256, num_heads=2, mlp_ratio=2,
                                                       in_channels=3, patch_size=4, spatial_merge_size=2,
                                                       temporal_patch_size=2),
                                 "mrope_section": [8, 12, 12], "image_token_id": 2000, "video_token_id": 2001,
                                 "vision_start_token_id": 2002}),
    "tiny-qwen2.5-vl": dict(model_type="qwen2_5_vl", vocab_size=2048, hidden_size=256, intermediate_size=512,
                            num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, rope_theta=1e6, eos_token_id=2,
                            extra={"vision_config": dict(depth=3, hidden_size=64, out_hidden_size=256, intermediate_size=96,
                                                         num_heads=2, in_channels=3, patch_size=4, spatial_merge_size=2,
                                                         temporal_patch_size=2, window_size=16, fullatt_block_indexes=[1],
                                                         hidden_act="silu"),
                                   "mrope_section": [8, 12, 12], "image_token_id": 2000, "video_token_id": 2001,
                                   "vision_start_token_id": 2002}),
    "tiny-qwen3-vl": dict(model_type="qwen3_vl", vocab_size=2048, hidden_size=256, intermediate_size=512,
                          num_hidden_layers=4, num_attention_heads=4, num_key_value_heads=2, head_dim=64, rope_theta=5e6,
                          eos_token_id=2,
                          extra={"vision_config": dict(depth=4, hidden_size=64, out_hidden_size=256, intermediate_size=96,
                                                       num_heads=2, in_channels=3, patch_size=4, spatial_merge_size=2,
                                                       temporal_patch_size=2, num_position_embeddings=64,
                                                       deepstack_visual_indexes=[0, 2], hidden_act="gelu_pytorch_tanh"),
                                 "mrope_section": [12, 10, 10], "mrope_interleaved": True, "image_token_id": 2000,
                                 "video_token_id": 2001, "vision_start_token_id": 2002}),
    "tiny-qwen3-vl-moe": dict(model_type="qwen3_vl_moe", vocab_size=2048, hidden_size=256, intermediate_size=512,
                              num_hidden_layers=3, num_attention_heads=4, num_key_value_heads=2, head_dim=64, rope_theta=5e6,
                              num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128, eos_token_id=2,
                              extra={"vision_config": dict(depth=3, hidden_size=64, out_hidden_size=256, intermediate_size=96,
                                                           num_heads=2, in_channels=3, patch_size=4, spatial_merge_size=2,
                                                           temporal_patch_size=2, num_position_embeddings=64,
                                                           deepstack_visual_indexes=[0, 1], hidden_act="gelu_pytorch_tanh"),
                                     "mrope_section": [12, 10, 10], "mrope_interleaved": True, "image_token_id": 2000,
                                     "video_token_id": 2001, "vision_start_token_id": 2002}),
    "qwen3-vl-30b-a3b": dict(model_type="qwen3_vl_moe", vocab_size=151936, hidden_size=2048, intermediate_size=6144,
                             num_hidden_layers=48, num_attention_heads=32, num_key_value_heads=4, head_dim=128, rope_theta=5e6,
                             num_experts=128, num_experts_per_tok=8, moe_intermediate_size=768, eos_token_id=151645,
                             max_position_embeddings=262144,
                             extra={"vision_config": dict(depth=27, hidden_size=1152, out_hidden_size=2048,
                                                          intermediate_size=4304, num_heads=16, in_channels=3, patch_size=16,
                                                          spatial_merge_size=2, temporal_patch_size=2,
                                                          num_position_embeddings=2304, deepstack_visual_indexes=[8, 16, 24],
                                                          hidden_act="gelu_pytorch_tanh"),
                                    "mrope_section": [24, 20, 20], "mrope_interleaved": True, "image_token_id": 151655,
                                    "video_token_id": 151656, "vision_start_token_id": 151652}),
    "qwen3-vl-8b": dict(model_type="qwen3_vl", vocab_size=151936, hidden_size=4096, intermediate_size=12288,
                        num_hidden_layers=36, num_attention_heads=32, num_key_value_heads=8, head_dim=128, rope_theta=5e6,
                        eos_token_id=151645, max_position_embeddings=262144,
                        extra={"vision_config": dict(depth=27, hidden_size=1152, out_hidden_size=4096, intermediate_size=4304,
                                                     num_heads=16, in_channels=3, patch_size=16, spatial_merge_size=2,
                                                     temporal_patch_size=2, num_position_embeddings=2304,
                                                     deepstack_visual_indexes=[8, 16, 24], hidden_act="gelu_pytorch_tanh"),
                               "mrope_section": [24, 20, 20], "mrope_interleaved": True, "image_token_id": 151655,
                               "video_token_id": 151656, "vision_start_token_id": 151652}),
    "qwen2.5-vl-7b": dict(model_type="qwen2_5_vl", vocab_size=152064, hidden_size=3584, intermediate_size=18944,
                          num_hidden_layers=28, num_attention_heads=28, num_key_value_heads=4, rope_theta=1e6,
                          eos_token_id=151645,
                          extra={"vision_config": dict(depth=32, hidden_size=1280, out_hidden_size=3584, intermediate_size=3420,
                                                       num_heads=16, in_channels=3, patch_size=14, spatial_merge_size=2,
                                                       temporal_patch_size=2, window_size=112,
                                                       fullatt_block_indexes=[7, 15, 23, 31], hidden_act="silu"),
                                 "mrope_section": [16, 24, 24], "image_token_id": 151655, "video_token_id": 151656,
                                 "vision_start_token_id": 151652}),
    "qwen2-vl-7b": dict(model_type="qwen2_vl", vocab_size=152064, hidden_size=3584, intermediate_size=18944,
                        num_hidden_layers=28, num_attention_heads=28, num_key_value_heads=4, rope_theta=1e6,
                        eos_token_id=151645,
                        extra={"vision_config": dict(depth=32, embed_dim=1280, hidden_size=3584, num_heads=16, mlp_ratio=4,
                                                     in_channels=3, patch_size=14, spatial_merge_size=2,
                                                     temporal_patch_size=2),
                               "mrope_section": [16, 24, 24], "image_token_id": 151655, "video_token_id": 151656,
                               "vision_start_token_id": 151652}),
    "tiny-apertus": dict(model_type="apertus", vocab_size=2048, hidden_size=256, intermediate_size=512, num_hidden_layers=2,
                         num_attention_heads=4, num_key_value_heads=2, rope_theta=1e6, rms_norm_eps=1e-5, eos_token_id=2),
    "apertus-8b": dict(model_type="apertus", vocab_size=131072, hidden_size=4096, intermediate_size=21504,
                       num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8, rope_theta=1.2e7,
                       rms_norm_eps=1e-5, eos_token_id=2, max_position_embeddings=65536,
                       extra={"rope_scaling": {"rope_type": "llama3", "factor": 8.0, "original_max_position_embeddings": 8192,
                                               "low_freq_factor": 1.0, "high_freq_factor": 4.0}}),
    "tiny-fuganex": dict(model_type="fuganex", vocab_size=640, hidden_size=192, eos_token_id=2, rms_norm_eps=1e-6,
                         layer_specs=_fuganex_specs(1, 6, 2, 32, 40, 6, 320, 6, 3, 32)),
    # real-model sizes for benchmarks: the widths of llama-3-8b, a third of the layers with windowed attention
    "fuganex-8b": dict(model_type="fuganex", vocab_size=128256, hidden_size=4096, eos_token_id=None, rms_norm_eps=1e-5,
                       num_attention_heads=32, num_key_value_heads=8, head_dim=128, intermediate_size=14336,
                       layer_specs=_fuganex_specs(10, 32, 8, 128, 1024, 4, 14336, 32, 16, 128)),
    "tiny-padodra": dict(model_type="padodra", vocab_size=704, hidden_size=160, eos_token_id=2, rms_norm_eps=1e-6,
                         embedding_scale=4.0, logit_scale=0.5,
                         layer_specs=_padodra_specs(1, 4, 2, 48, 56, 288, (4, 32, 16, 40, 56))),
    # real-model sizes for benchmarks: the widths of llama-3-8b, chunks of 2048, a rank of 512 in every third layer
    "padodra-8b": dict(model_type="padodra", vocab_size=128256, hidden_size=4096, eos_token_id=None, rms_norm_eps=1e-5,
                       num_attention_heads=32, num_key_value_heads=8, head_dim=128, intermediate_size=14336,
                       layer_specs=_padodra_specs(10, 32, 8, 128, 2048, 14336, (32, 128, 64, 128, 512))),
    "tiny-golonex": dict(model_type="golonex", vocab_size=600, hidden_size=144, eos_token_id=2, rms_norm_eps=1e-6,
                         logit_softcap=20.0, side_dim=16,
                         layer_specs=_golonex_specs(1, 6, 3, 32, 50, (168, 3, 4), (4, 24, 16, 40, 64, 72), (6, 2, 104, 88))),
    # real-model sizes for benchmarks: the widths of llama-3-8b, windows of 1024, its feed-forward cut into 16 experts
    "golonex-8b": dict(model_type="golonex", vocab_size=128256, hidden_size=4096, eos_token_id=None, rms_norm_eps=1e-5,
                       num_attention_heads=32, num_key_value_heads=8, head_dim=128, intermediate_size=896, logit_softcap=30.0,
                       side_dim=256,
                       layer_specs=_golonex_specs(10, 32, 8, 128, 1024, (4096, 16, 4), (32, 128, 64, 128, 512, 1536),
                                                  (16, 4, 896, 3584))),
    "tiny-malinex": dict(model_type="malinex", vocab_size=616, hidden_size=136, eos_token_id=2, rms_norm_eps=1e-6, logit_scale=0.5,
                         max_position_embeddings=1024,
                         layer_specs=_malinex_specs(2, 6, 3, 24, (3, 24, 40, 8.0, 8), 296, (6, 2, 72, 104))),
    # real-model sizes for benchmarks: the widths of llama-3-8b, its feed-forward cut into 16 experts
    "malinex-8b": dict(model_type="malinex", vocab_size=128256, hidden_size=4096, eos_token_id=None, rms_norm_eps=1e-5,
                       num_attention_heads=32, num_key_value_heads=8, head_dim=128, intermediate_size=896,
                       max_position_embeddings=32768,
                       layer_specs=_malinex_specs(10, 32, 8, 128, (32, 128, 128, 16.0, 16), 14336, (16, 4, 896, 3584))),
    "llama-3-8b": dict(model_type="llama", vocab_size=128256, hidden_size=4096, intermediate_size=14336,
                       num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8, rope_theta=5e5,
                       rms_norm_eps=1e-5, eos_token_id=128001),
}


def preset(name: str, **overrides) -> ModelConfig:
    kw = dict(PRESETS[name])
    kw.update(overrides)
    return ModelConfig(**kw)
