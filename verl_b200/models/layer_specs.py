"""Per-layer descriptions of decoders whose layers differ from one another (``ModelConfig.layer_specs``).

A layer is a mixer (softmax attention, latent attention or a gated delta rule, each with its own sizes) and an optional
feed-forward. The specs carry every size and constant of a mechanism, so that another design can combine them differently;
what a design fixes instead of writing it in its config.json is in ``DESIGNS``."""

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
    """Softmax attention. ``window`` (0 = full causal): a query sees the last ``window`` positions, its own included, and
    the first ``keep_first`` positions of the sequence. ``chunk`` (0 = none): a query sees the keys of its own chunk of
    ``chunk`` positions, counted from the start of the sequence. ``bias_rows`` / ``bias_max``: learned distance
    bias per head, added to the scaled score (``bias_rows`` 0 = none); see :func:`distance_buckets`. ``softcap`` > 0: scaled
    scores become ``softcap * tanh(score / softcap)``. ``sink``: a learned number per head whose exponential joins the
    softmax denominator. ``gate``: the heads are multiplied with the sigmoid of a projection of the mixer's input."""

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
    gate: bool = False

    @property
    def q_size(self) -> int:
        return self.heads * self.dim

    @property
    def k_size(self) -> int:
        return self.kv_heads * self.dim

    @property
    def v_size(self) -> int:
        return self.kv_heads * self.vdim

    @property
    def out_size(self) -> int:
        return self.heads * self.vdim

    @property
    def proj_size(self) -> int:
        """q | k | v (| output gate)."""
        return self.q_size + self.k_size + self.v_size + (self.out_size if self.gate else 0)

    @property
    def norm_sizes(self) -> tuple[int, int]:
        """Weights of the query and of the key norm."""
        return {None: (0, 0), "projection": (self.q_size, self.k_size), "head": (self.dim, self.dim)}[self.qk_norm]


@dataclass(frozen=True)
class LatentSpec:
    """Latent attention: every head's keys (their unrotated ``dim``) and values are projections of one normed latent of
    ``kv_rank`` numbers per token; ``rot_dim`` rotated key dimensions are shared by all heads. Latent and rotated part are
    what the cache holds. Full causal. ``gate`` as in :class:`AttentionSpec`."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rotary: RotarySpec
    gate: bool = False

    @property
    def q_size(self) -> int:
        return self.heads * (self.dim + self.rot_dim)

    @property
    def latent_size(self) -> int:
        """Latent and rotated part of one token."""
        return self.kv_rank + self.rot_dim

    @property
    def out_size(self) -> int:
        return self.heads * self.vdim

    @property
    def proj_size(self) -> int:
        """q | latent, rotated key (| output gate)."""
        return self.q_size + self.latent_size + (self.out_size if self.gate else 0)

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
class GluSpec:
    """Gated linear unit. ``act`` "clamped": ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``,
    ``g * sigmoid(alpha * g) * (u + 1)``; "gelu_tanh": ``gelu(gate) * up`` with the tanh form of gelu."""

    ff: int
    limit: float = 0.0
    alpha: float = 1.702
    act: str = "clamped"


@dataclass(frozen=True)
class Design:
    """What a design fixes for all its models. ``norm``: "pre" (a sublayer reads the normed stream, its output is added as it
    is) or "post" (it reads the stream, its normed output is added). ``mask``: what an attention layer's mask size means."""

    norm: str = "pre"
    mask: str = "window"
    qk_norm: Optional[str] = "projection"
    interleaved: bool = False  # rotary layout of attention layers (latent attention: always halves)
    sink: bool = False
    gate: bool = False
    act: str = "clamped"
    logit_scale: bool = False  # config.json has a factor for the logits


DESIGNS: dict[str, Design] = {
    "fuganex": Design(),
    "padodra": Design(norm="post", mask="chunk", qk_norm="head", interleaved=True, sink=True, gate=True, act="gelu_tanh",
                      logit_scale=True),
}
_KINDS = {AttentionSpec: "attention", LatentSpec: "latent_attention", DeltaSpec: "delta"}


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, LatentSpec, DeltaSpec]
    mlp: Optional[GluSpec] = None

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
                                  softcap=float(m.get("softcap") or 0.0), sink=design.sink, gate=design.gate)
            if mixer.rotary is not None and mixer.rotary.dims > mixer.dim:
                raise ValueError(f"{mixer.rotary.dims} rotated dimensions in heads of {mixer.dim}")
        elif d["type"] == "latent_attention":
            mixer = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                               float(m["scale"]), RotarySpec.from_dict(m["rot"], False), design.gate)
            if mixer.rotary.dims != mixer.rot_dim:
                raise ValueError(f"{mixer.rotary.dims} rotated dimensions in a rotated part of {mixer.rot_dim}")
        elif d["type"] == "delta":
            mixer = DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        else:
            raise ValueError(f"unknown layer type {d['type']!r} (known: {', '.join(_KINDS.values())})")
        if mixer.heads % getattr(mixer, "kv_heads", 1):
            raise ValueError(f"{mixer.heads} heads are not a multiple of {mixer.kv_heads} key/value heads")
        mlp = d.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r} (known: dense)")
            mlp = GluSpec(int(mlp["ff"]), float(mlp["limit"]) if design.act == "clamped" else 0.0, act=design.act)
        return cls(mixer, mlp)

    def to_dict(self) -> dict[str, Any]:
        m = self.mixer
        if self.kind == "attention":
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.chunk:
                mix["mask"] = {"size": m.chunk}
            elif m.window or m.keep_first:
                mix["mask"] = {"size": m.window, "keep_first": m.keep_first}
            if m.bias_max:
                mix["bias_max"] = int(m.bias_max) if m.bias_max == int(m.bias_max) else m.bias_max
            if m.rotary is not None:
                mix["rot"] = m.rotary.to_dict()
            if m.softcap:
                mix["softcap"] = m.softcap
        elif self.kind == "latent_attention":
            mix = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                   "scale": m.scale, "rot": m.rotary.to_dict()}
        else:
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
        mlp = None
        if self.mlp is not None:
            mlp = {"kind": "dense", "ff": self.mlp.ff}
            if self.mlp.act == "clamped":
                mlp["limit"] = self.mlp.limit
        return {"type": self.kind, "mixer": mix, "mlp": mlp}

    def with_bias_rows(self, rows: int) -> "LayerSpec":
        return replace(self, mixer=replace(self.mixer, bias_rows=int(rows)))

    def num_parameters(self, width: int) -> int:
        m = self.mixer
        n = width + width * (m.proj_size + m.out_size)  # norm1, projections
        if self.kind == "attention":
            n += m.bias_rows * m.heads + sum(m.norm_sizes) + (m.heads if m.sink else 0)
        elif self.kind == "latent_attention":
            n += m.kv_rank + m.up_size * m.kv_rank
        else:
            n += m.channels * m.conv + 2 * m.heads + m.vdim
        if self.mlp is not None:
            n += width + 3 * width * self.mlp.ff
        return n


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
