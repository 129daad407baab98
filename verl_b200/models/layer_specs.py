"""Per-layer descriptions of decoders whose layers differ from one another (``ModelConfig.layer_specs``).

A layer is a mixer (softmax attention or a gated delta rule, each with its own sizes) and an optional feed-forward. The
specs carry every size and constant of a mechanism, so that another design can combine them differently."""

from __future__ import annotations

import math
from dataclasses import dataclass, replace
from fractions import Fraction
from typing import Any, Optional, Union


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention without rotation. ``window`` (0 = full causal): a query sees the last ``window`` positions, its
    own included, and the first ``keep_first`` positions of the sequence. ``bias_rows`` / ``bias_max``: learned distance
    bias per head, added to the scaled score (``bias_rows`` 0 = none); see :func:`distance_buckets`."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    keep_first: int = 0
    bias_max: float = 0.0
    bias_rows: int = 0
    qk_norm: bool = True  # RMS norm over the whole query (key) projection, before the split into heads

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
    """Clamped gated linear unit: ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``,
    ``g * sigmoid(alpha * g) * (u + 1)``."""

    ff: int
    limit: float
    alpha: float = 1.702


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, DeltaSpec]
    mlp: Optional[GluSpec] = None

    @property
    def kind(self) -> str:
        return "attention" if isinstance(self.mixer, AttentionSpec) else "delta"

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "LayerSpec":
        """One entry of the ``layers`` list of a config.json."""
        m = d["mixer"]
        if d["type"] == "attention":
            mask = m.get("mask") or {}
            mixer = AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                  int(mask.get("size") or 0), int(mask.get("keep_first") or 0),
                                  float(m.get("bias_max") or 0.0))
        elif d["type"] == "delta":
            mixer = DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        else:
            raise ValueError(f"unknown layer type {d['type']!r} (known: attention, delta)")
        if mixer.heads % mixer.kv_heads:
            raise ValueError(f"{mixer.heads} heads are not a multiple of {mixer.kv_heads} key/value heads")
        mlp = d.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r} (known: dense)")
            mlp = GluSpec(int(mlp["ff"]), float(mlp["limit"]))
        return cls(mixer, mlp)

    def to_dict(self) -> dict[str, Any]:
        m = self.mixer
        if self.kind == "attention":
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                   "bias_max": int(m.bias_max) if m.bias_max == int(m.bias_max) else m.bias_max,
                   "mask": {"size": m.window, "keep_first": m.keep_first}}
        else:
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
        mlp = None if self.mlp is None else {"kind": "dense", "ff": self.mlp.ff, "limit": self.mlp.limit}
        return {"type": self.kind, "mixer": mix, "mlp": mlp}

    def with_bias_rows(self, rows: int) -> "LayerSpec":
        return replace(self, mixer=replace(self.mixer, bias_rows=int(rows)))

    def num_parameters(self, width: int) -> int:
        m = self.mixer
        n = width  # norm1
        if self.kind == "attention":
            n += width * (m.q_size + m.k_size + m.v_size + m.out_size) + m.bias_rows * m.heads
            n += m.q_size + m.k_size if m.qk_norm else 0
        else:
            n += width * (m.proj_size + m.out_size) + m.channels * m.conv + 2 * m.heads + m.vdim
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
