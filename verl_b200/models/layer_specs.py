"""Per-layer descriptions of decoders whose layers differ from one another (``ModelConfig.layer_specs``).

A layer is a mixer (attention, latent attention, a gated delta rule, gated linear attention or a gated linear recurrent unit,
each with its own sizes) and an optional feed-forward (two matrices, a gated linear unit or a mixture of either). The specs carry
every size and constant of a mechanism, so that another design can combine them differently; what a design fixes instead of
writing it in its config.json is in ``DESIGNS``."""

from __future__ import annotations

import math
from dataclasses import dataclass, replace
from fractions import Fraction
from typing import Any, Optional, Union


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first ``dims`` dimensions of a vector: pair i turns by ``position * f_i`` with
    ``f_i = base ** (-2 i / dims)``. ``interleaved``: pair i is (2 i, 2 i + 1), else (i, i + dims / 2). ``scaling``: the items
    of a frequency scaling, told apart by their keys: ``low`` / ``high`` = wavelength bands (Llama 3.1), ``fast`` /
    ``slow`` = a ramp over the pair index (YaRN, which also scales cos and sin)."""

    dims: int
    base: float
    interleaved: bool = False
    scaling: tuple = ()

    @classmethod
    def from_dict(cls, d: dict[str, Any], interleaved: bool) -> "RotarySpec":
        spec = cls(int(d["dims"]), float(d["base"]), interleaved, tuple(sorted((d.get("scaling") or {}).items())))
        keys = {k for k, _ in spec.scaling}
        if spec.dims % 2:
            raise ValueError(f"rotary positions need an even number of dimensions, got {spec.dims}")
        if keys and not ({"factor", "original"} <= keys and ({"low", "high"} <= keys or {"fast", "slow"} <= keys)):
            raise ValueError(f"unknown frequency scaling with the keys {sorted(keys)}")
        return spec

    def to_dict(self) -> dict[str, Any]:
        return {"dims": self.dims, "base": self.base, **({"scaling": dict(self.scaling)} if self.scaling else {})}

    def frequencies(self) -> list[float]:
        """``dims / 2`` angular frequencies (double precision)."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        c = dict(self.scaling)
        if "low" in c:
            def scaled(x):
                wave = 2 * math.pi / x
                if wave < c["original"] / c["high"]:
                    return x
                if wave > c["original"] / c["low"]:
                    return x / c["factor"]
                s = (c["original"] / wave - c["low"]) / (c["high"] - c["low"])
                return (1 - s) * x / c["factor"] + s * x

            return [scaled(x) for x in f]
        if "fast" in c:
            def dim_at(turns):
                return self.dims * math.log(c["original"] / (turns * 2 * math.pi)) / (2 * math.log(self.base))

            lo = max(math.floor(dim_at(c["fast"])), 0)
            hi = min(math.ceil(dim_at(c["slow"])), self.dims - 1)
            ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
            return [x / c["factor"] * r + x * (1 - r) for x, r in zip(f, ramp)]
        return f

    @property
    def amplitude(self) -> float:
        """Factor of cos and sin."""
        c = dict(self.scaling)
        return 0.1 * math.log(c["factor"]) + 1.0 if "fast" in c else 1.0


@dataclass(frozen=True)
class AttentionSpec:
    """Attention. ``window`` (0 = full causal): a query sees the last ``window`` positions, its own included, and
    the first ``keep_first`` positions of the sequence. ``chunk`` (0 = none): a query sees the keys of its own chunk of
    ``chunk`` positions, counted from the start of the sequence. ``bias_rows`` / ``bias_max``: learned distance
    bias per head, added to the scaled score (``bias_rows`` 0 = none); see :func:`distance_buckets`. ``softcap`` > 0: scaled
    scores become ``softcap * tanh(score / softcap)``. ``sink``: a learned number per head whose exponential joins the
    softmax denominator. ``gate``: the heads are multiplied with the sigmoid of a projection of the mixer's input, element by
    element ("element") or one number per head ("head"). ``key_values``: no value projection, the unrotated key serves as the
    value too. ``qkv_bias``: the projections have biases. ``q_temp`` (coef, every): queries at position p are multiplied by
    1 + coef ln(floor((p + 1) / every) + 1). ``log_bias``: r1 ln(1 + r2 (i - j)) is taken off the scaled score, with two learned
    numbers per head. ``weighting`` "sigmoid": a key weighs the sigmoid of its score plus a learned number of the head, whatever
    the other keys have; "softmax": as usual."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    keep_first: int = 0
    bias_max: float = 0.0
    bias_rows: int = 0
    # RMS norm of queries and keys: None, "projection" (over all heads at once) or "head" (each head, one weight for all)
    qk_norm: Optional[str] = "projection"
    rotary: Optional[RotarySpec] = None
    chunk: int = 0
    softcap: float = 0.0
    sink: bool = False
    gate: Optional[str] = None
    key_values: bool = False
    qkv_bias: bool = False
    q_temp: Optional[tuple] = None
    log_bias: bool = False
    weighting: str = "softmax"

    @property
    def q_size(self) -> int:
        return self.heads * self.dim

    @property
    def k_size(self) -> int:
        return self.kv_heads * self.dim

    @property
    def v_size(self) -> int:
        """Rows of the value projection."""
        return 0 if self.key_values else self.kv_heads * self.vdim

    @property
    def out_size(self) -> int:
        return self.heads * self.vdim

    @property
    def proj_size(self) -> int:
        """q | k | v (| output gate)."""
        return self.q_size + self.k_size + self.v_size + self.gate_size

    @property
    def gate_size(self) -> int:
        return {None: 0, "element": self.out_size, "head": self.heads}[self.gate]

    @property
    def head_numbers(self) -> int:
        """Learned numbers per head besides tables: sink, r1 and r2, the sigmoid's shift."""
        return int(self.sink) + 2 * int(self.log_bias) + int(self.weighting == "sigmoid")

    @property
    def norm_sizes(self) -> tuple[int, int]:
        """Weights of the query and of the key norm."""
        return {None: (0, 0), "projection": (self.q_size, self.k_size), "head": (self.dim, self.dim)}[self.qk_norm]


@dataclass(frozen=True)
class LatentSpec:
    """Latent attention: every head's keys (their unrotated ``dim``) and values are projections of one normed latent of
    ``kv_rank`` numbers per token; ``rot_dim`` rotated key dimensions are shared by all heads. Latent and rotated part are
    what the cache holds. ``q_rank`` > 0: the queries are projections of a normed latent of their own. ``window`` (0 = full
    causal) and ``sink`` as in :class:`AttentionSpec`; ``gate`` as there, or one number per head ("head")."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rotary: RotarySpec
    gate: Optional[str] = None
    q_rank: int = 0
    window: int = 0
    sink: bool = False

    @property
    def q_size(self) -> int:
        return self.heads * (self.dim + self.rot_dim)

    @property
    def q_in(self) -> int:
        """Rows of the input projection that the queries come from: the queries themselves, or their latent."""
        return self.q_rank or self.q_size

    @property
    def latent_size(self) -> int:
        """Latent and rotated part of one token."""
        return self.kv_rank + self.rot_dim

    @property
    def out_size(self) -> int:
        return self.heads * self.vdim

    @property
    def gate_size(self) -> int:
        return {None: 0, "element": self.out_size, "head": self.heads}[self.gate]

    @property
    def proj_size(self) -> int:
        """q or its latent | latent, rotated key (| output gate)."""
        return self.q_in + self.latent_size + self.gate_size

    @property
    def up_size(self) -> int:
        """Keys and values out of the latent."""
        return self.heads * (self.dim + self.vdim)


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule with short convolutions of ``conv`` taps on q, k and v."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @property
    def channels(self) -> int:
        """Convolved channels: q | k | v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def proj_size(self) -> int:
        """q | k | v | output gate | b | a."""
        return self.channels + self.heads * self.vdim + 2 * self.heads

    @property
    def out_size(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class GlaSpec:
    """Gated linear attention: a state [dim, vdim] per head whose row d decays by sigmoid(z_d) ** (1 / tau) before k v^T is added;
    the head's output S^T q (q scaled by dim ** -0.5) is RMS-normed and multiplied with the silu of a gate. z comes from the
    mixer's input through ``rank`` numbers (0: not known yet, the weights' shapes give it)."""

    heads: int
    dim: int
    vdim: int
    tau: float = 16.0
    rank: int = 0

    @property
    def qk_size(self) -> int:
        return self.heads * self.dim

    @property
    def proj_size(self) -> int:
        """q | k | v | output gate | decay's first matrix."""
        return 2 * self.qk_size + 2 * self.out_size + self.rank

    @property
    def out_size(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class LruSpec:
    """Griffin's RG-LRU block. One branch is a gelu; the other is a short convolution of ``conv`` taps, giving u, and a diagonal
    recurrence per channel: S decays by a = exp(-power * softplus(lam) * r) and takes in i * u, scaled by sqrt(1 - a * a). Decay
    gate r and input gate i are sigmoids of u times block-diagonal matrices of ``blocks`` blocks. The branches are multiplied."""

    width: int
    blocks: int
    conv: int
    power: float = 8.0

    @property
    def block_size(self) -> int:
        return self.width // self.blocks

    @property
    def proj_size(self) -> int:
        """gelu branch | recurrent branch."""
        return 2 * self.width

    @property
    def out_size(self) -> int:
        return self.width


@dataclass(frozen=True)
class GluSpec:
    """Gated linear unit. ``act`` "clamped": ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``,
    ``g * sigmoid(alpha * g) * (u + 1)``; "gelu_tanh": ``gelu(gate) * up`` with the tanh form of gelu; "silu":
    ``silu(gate) * up``."""

    ff: int
    limit: float = 0.0
    alpha: float = 1.702
    act: str = "clamped"

    def num_parameters(self, width: int) -> int:
        return 3 * width * self.ff


@dataclass(frozen=True)
class MlpSpec:
    """Two matrices with an activation between them: "gelu" (the exact form, with erf) or "relu2" (the square of relu)."""

    ff: int
    act: str = "gelu"

    def num_parameters(self, width: int) -> int:
        return 2 * width * self.ff


@dataclass(frozen=True)
class MoeSpec:
    """Mixture of ``experts`` units of ``ff``, ``top`` of them per token: gated linear units, or without ``gated`` two matrices.
    Router scores: "sigmoid" or "softmax" of the logits, computed in fp32; the ``top`` largest (``correction``: the largest after a
    learned number per expert is added, for the choice alone) are chosen and weigh as they are (``renormalize``: divided by
    their sum). ``weigh`` "input": an expert runs on its weight times the token, "output": its result is multiplied.
    ``shared_ff`` > 0: a unit of that size runs for every token; ``shared_gate``: its result is multiplied with the sigmoid of a
    projection to one number."""

    experts: int
    top: int
    ff: int
    shared_ff: int = 0
    act: str = "silu"
    score: str = "sigmoid"
    renormalize: bool = False
    weigh: str = "input"
    gated: bool = True
    correction: bool = False
    shared_gate: bool = True

    @property
    def router_rows(self) -> int:
        """Router | gate of the shared unit."""
        return self.experts + (1 if self.shared_ff and self.shared_gate else 0)

    @property
    def shared(self) -> Union[GluSpec, MlpSpec, None]:
        """The unit that runs for every token."""
        if not self.shared_ff:
            return None
        return GluSpec(self.shared_ff, act=self.act) if self.gated else MlpSpec(self.shared_ff, self.act)

    def num_parameters(self, width: int) -> int:
        matrices = 3 if self.gated else 2
        return (width * (self.router_rows + matrices * (self.experts * self.ff + self.shared_ff))
                + (self.experts if self.correction else 0))


@dataclass(frozen=True)
class Design:
    """What a design fixes for all its models. ``norm``: "pre" (a sublayer reads the normed stream, its output is added as it
    is), "post" (it reads the stream, its normed output is added) or "both" (it reads the normed stream, its normed output is
    added). ``mask``: what an attention layer's mask size means."""

    norm: str = "pre"
    mask: str = "window"
    qk_norm: Optional[str] = "projection"
    interleaved: bool = False  # rotary layout of attention layers
    sink: bool = False
    gate: Optional[str] = None
    key_values: bool = False
    latent_interleaved: bool = False  # the same of latent attention
    latent_sink: bool = False
    latent_gate: Optional[str] = None
    qkv_bias: bool = False
    log_bias: bool = False
    weighting: str = "softmax"
    act: str = "clamped"       # of dense feed-forwards; "gelu" and "relu2" are two matrices, the others gated linear units
    expert_act: str = "silu"   # of mixtures
    score: str = "sigmoid"     # of routers
    renormalize: bool = False
    weigh: str = "input"
    correction: bool = False
    shared_gate: bool = True
    residual_gate: bool = False  # a sublayer's result times the sigmoid of a projection of what it reads
    embedding: str = "scale"   # "scale": times a factor of config.json, "norm": RMS norm, "positions": plus a learned position
    tied: bool = False         # the embedding table is the output projection
    logit_scale: bool = False  # config.json has a factor for the logits
    logit_softcap: bool = False  # config.json has a soft cap for the logits
    side: bool = False         # layers add an input of their own per token (config.json: its size)


DESIGNS: dict[str, Design] = {
    "fuganex": Design(),
    "padodra": Design(norm="post", mask="chunk", qk_norm="head", interleaved=True, sink=True, gate="element",
                      latent_gate="element", act="gelu_tanh", logit_scale=True),
    "golonex": Design(qk_norm=None, interleaved=True, key_values=True, latent_interleaved=True, latent_sink=True,
                      latent_gate="head", act="silu", embedding="norm", tied=True, logit_softcap=True, side=True),
    "malinex": Design(norm="both", gate="head", qkv_bias=True, log_bias=True, weighting="sigmoid", act="gelu", expert_act="relu2",
                      score="softmax", renormalize=True, weigh="output", correction=True, shared_gate=False, residual_gate=True,
                      embedding="positions", logit_scale=True),
}
PLAIN_ACTS = ("gelu", "relu2")  # of feed-forwards of two matrices
_KINDS = {AttentionSpec: "attention", LatentSpec: "latent_attention", DeltaSpec: "delta", GlaSpec: "gla", LruSpec: "rglru"}


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, LatentSpec, DeltaSpec, GlaSpec, LruSpec]
    mlp: Union[GluSpec, MlpSpec, MoeSpec, None] = None
    weights_of: Optional[int] = None  # the layer whose weights this one uses, with a cache or state of its own

    @property
    def kind(self) -> str:
        return _KINDS[type(self.mixer)]

    @classmethod
    def from_dict(cls, d: dict[str, Any], design: Design) -> "LayerSpec":
        """One entry of the ``layers`` list of a config.json."""
        m = d["mixer"]
        if d["type"] == "attention":
            mask, size = m.get("mask") or {}, int((m.get("mask") or {}).get("size") or 0)
            chunked = design.mask == "chunk"
            mixer = AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                  0 if chunked else size, int(mask.get("keep_first") or 0), float(m.get("bias_max") or 0.0),
                                  qk_norm=design.qk_norm, chunk=size if chunked else 0,
                                  rotary=RotarySpec.from_dict(m["rot"], design.interleaved) if m.get("rot") else None,
                                  softcap=float(m.get("softcap") or 0.0), sink=design.sink, gate=design.gate,
                                  key_values=design.key_values, qkv_bias=design.qkv_bias, log_bias=design.log_bias,
                                  weighting=design.weighting,
                                  q_temp=(float(m["q_temp"]["coef"]), float(m["q_temp"]["every"])) if m.get("q_temp") else None)
            if mixer.q_temp is not None and not mixer.q_temp[1] > 0:
                raise ValueError(f"query temperature in steps of {mixer.q_temp[1]}")
            if mixer.rotary is not None and mixer.rotary.dims > mixer.dim:
                raise ValueError(f"{mixer.rotary.dims} rotated dimensions in heads of {mixer.dim}")
            if mixer.key_values and mixer.vdim != mixer.dim:
                raise ValueError(f"values of {mixer.vdim} that are the keys of {mixer.dim}")
        elif d["type"] == "latent_attention":
            mixer = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                               float(m["scale"]), RotarySpec.from_dict(m["rot"], design.latent_interleaved),
                               design.latent_gate, int(m.get("q_rank") or 0), int((m.get("mask") or {}).get("size") or 0),
                               design.latent_sink)
            if mixer.rotary.dims != mixer.rot_dim:
                raise ValueError(f"{mixer.rotary.dims} rotated dimensions in a rotated part of {mixer.rot_dim}")
        elif d["type"] == "delta":
            mixer = DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        elif d["type"] == "gla":
            mixer = GlaSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]))
        elif d["type"] == "rglru":
            mixer = LruSpec(int(m["width"]), int(m["blocks"]), int(m["conv"]))
            if mixer.width % mixer.blocks:
                raise ValueError(f"a width of {mixer.width} is not a multiple of {mixer.blocks} blocks")
        else:
            raise ValueError(f"unknown layer type {d['type']!r} (known: {', '.join(_KINDS.values())})")
        if getattr(mixer, "heads", 0) % getattr(mixer, "kv_heads", 1):
            raise ValueError(f"{mixer.heads} heads are not a multiple of {mixer.kv_heads} key/value heads")
        mlp = d.get("mlp")
        if mlp is not None:
            kind = mlp.get("kind", "dense")
            if kind == "moe" and (design.act == design.expert_act or design.expert_act in PLAIN_ACTS):
                mlp = MoeSpec(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]),
                              int((mlp.get("shared") or {}).get("ff") or 0), design.expert_act, design.score,
                              design.renormalize, design.weigh, design.expert_act not in PLAIN_ACTS, design.correction,
                              design.shared_gate)
                if not 0 < mlp.top <= mlp.experts:
                    raise ValueError(f"{mlp.top} of {mlp.experts} experts")
            elif kind == "dense" and design.act in PLAIN_ACTS:
                mlp = MlpSpec(int(mlp["ff"]), design.act)
            elif kind == "dense":
                mlp = GluSpec(int(mlp["ff"]), float(mlp["limit"]) if design.act == "clamped" else 0.0, act=design.act)
            else:
                raise ValueError(f"unknown feed-forward kind {kind!r} (known: dense, and moe where the design has experts)")
        of = d.get("weights_of")
        return cls(mixer, mlp, None if of is None else int(of))

    def to_dict(self) -> dict[str, Any]:
        m = self.mixer
        if self.kind == "attention":
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.chunk:
                mix["mask"] = {"size": m.chunk}
            elif m.window or m.keep_first:
                mix["mask"] = {"size": m.window, **({"keep_first": m.keep_first} if m.keep_first or not m.key_values else {})}
            if m.bias_max:
                mix["bias_max"] = int(m.bias_max) if m.bias_max == int(m.bias_max) else m.bias_max
            if m.rotary is not None:
                mix["rot"] = m.rotary.to_dict()
            if m.softcap:
                mix["softcap"] = m.softcap
            if m.q_temp is not None:
                mix["q_temp"] = {"coef": m.q_temp[0], "every": int(m.q_temp[1]) if m.q_temp[1] == int(m.q_temp[1]) else m.q_temp[1]}
        elif self.kind == "latent_attention":
            mix = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                   "scale": m.scale, "rot": m.rotary.to_dict()}
            if m.q_rank:
                mix["q_rank"] = m.q_rank
            if m.window:
                mix["mask"] = {"size": m.window}
        elif self.kind == "gla":
            mix = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}
        elif self.kind == "rglru":
            mix = {"width": m.width, "blocks": m.blocks, "conv": m.conv}
        else:
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
        mlp = None
        if isinstance(self.mlp, MoeSpec):
            mlp = {"kind": "moe", "expert": {"ff": self.mlp.ff}, "router": {"experts": self.mlp.experts, "top": self.mlp.top}}
            if self.mlp.shared_ff:
                mlp["shared"] = {"ff": self.mlp.shared_ff}
        elif self.mlp is not None:
            mlp = {"kind": "dense", "ff": self.mlp.ff}
            if self.mlp.act == "clamped":
                mlp["limit"] = self.mlp.limit
        d = {"type": self.kind, "mixer": mix, "mlp": mlp}
        return d if self.weights_of is None else {**d, "weights_of": self.weights_of}

    def with_sizes(self, **sizes: int) -> "LayerSpec":
        """With sizes of the mixer that only the weights' shapes give."""
        return replace(self, mixer=replace(self.mixer, **sizes))

    def num_parameters(self, width: int, design: Optional[Design] = None) -> int:
        m = self.mixer
        if self.weights_of is not None:
            return 0
        n = width + width * (m.proj_size + m.out_size)  # norm1, projections
        if self.kind == "attention":
            n += m.bias_rows * m.heads + sum(m.norm_sizes) + m.head_numbers * m.heads
            n += m.q_size + m.k_size + m.v_size if m.qkv_bias else 0
        elif self.kind == "latent_attention":
            n += m.kv_rank + m.up_size * m.kv_rank + (m.heads if m.sink else 0)
            if m.q_rank:
                n += m.q_rank + m.q_size * m.q_rank
        elif self.kind == "gla":
            n += m.qk_size * (m.rank + 1) + m.vdim
        elif self.kind == "rglru":  # biases of the branches, convolution, gates, lam
            n += m.width * (2 + m.conv + 1 + 2 * (m.block_size + 1) + 1)
        else:
            n += m.channels * m.conv + 2 * m.heads + m.vdim
        if self.mlp is not None:
            n += width + self.mlp.num_parameters(width)
        if design is not None:  # what a design adds to every sublayer
            per = (width if design.norm == "both" else 0) + (width * (width + 1) if design.residual_gate else 0)
            n += per * (1 if self.mlp is None else 2)
        return n


def weight_owner(specs: tuple, i: int) -> int:
    """The layer whose weights layer i uses."""
    seen = set()
    while specs[i].weights_of is not None:
        j = specs[i].weights_of
        if not 0 <= j < len(specs) or i in seen:
            raise ValueError(f"layer {i} uses the weights of layer {j}")
        if type(specs[j].mixer) is not type(specs[i].mixer):
            raise ValueError(f"layer {i} ({specs[i].kind}) uses the weights of layer {j} ({specs[j].kind})")
        seen.add(i)
        i = j
    return i


def distance_buckets(rows: int, far: float) -> list[int]:
    """Row of a distance table with ``rows`` rows for the distances 0, 1, ..., ceil(far) (every larger distance has the
    last row): with h = rows // 2 a distance n < h has its own row; from h on the rows are logarithmic,
    h + floor((rows - h) ln(n / h) / ln(far / h)), at most rows - 1. The floor is decided on exact fractions,
    (n / h) ^ (rows - h) against (far / h) ^ k, so that no edge depends on the rounding of a logarithm."""
    h = rows // 2
    far = Fraction(far)
    if h < 1 or far <= h:
        raise ValueError(f"a distance table of {rows} rows needs its largest distance above {h}, got {float(far)}")
    m, ratio = rows - h, far / h
    # smallest distance that belongs to row h + k, k = 1 .. m - 1: compared as floats first, exactly where they are close
    out = []
    for n in range(math.ceil(far) + 1):
        if n < h:
            out.append(n)
            continue
        x = m * math.log(n / h) / math.log(ratio)
        k = math.floor(x)
        near = round(x)
        if abs(x - near) < 1e-6:
            k = near if Fraction(n, h) ** m >= ratio ** near else near - 1
        out.append(min(rows - 1, h + k))
    return out
