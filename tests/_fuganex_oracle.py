"""Plain, slow implementation of the Fuganex design on the CPU: the yardstick of ``test_fuganex_*.py``.

One function per mechanism, token by token and head by head where that is the definition, written from the equations
and sharing nothing with the package. ``weights`` maps checkpoint tensor names to tensors, ``cfg`` is the parsed
``config.json``. Everything runs in the dtype of the weights after ``to(dtype)`` (float32 or float64).
"""

from __future__ import annotations

import json
import math
import struct
from fractions import Fraction

import torch


def read_safetensors(path):
    raw = open(path, "rb").read()
    (n,) = struct.unpack("<Q", raw[:8])
    head = json.loads(raw[8:8 + n])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    out = {}
    for name, d in head.items():
        if name == "__metadata__":
            continue
        lo, hi = d["data_offsets"]
        buf = bytearray(raw[8 + n + lo:8 + n + hi])
        out[name] = torch.frombuffer(buf, dtype=kinds[d["dtype"]]).reshape(d["shape"])
    return out


def rms_norm(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(x):
    return x / (1 + torch.exp(-x))


def distance_bucket(n: int, rows: int, far) -> int:
    """Row of a distance table with ``rows`` rows for distance ``n``: exact below rows // 2, then logarithmic up to
    ``far``. The comparison (n / h) ^ m >= (far / h) ^ k is done on fractions, so that no bucket edge is rounded."""
    h = rows // 2
    if n < h:
        return n
    m = rows - h
    r, d = Fraction(n, h), Fraction(far) / h
    k = 0
    while k < m and r ** m >= d ** (k + 1):
        k += 1
    return min(rows - 1, h + k)


def visible(i: int, j: int, size: int, keep_first: int) -> bool:
    return j <= i and (i - j < size or j < keep_first)


def attention_scores(q, k, scale, rel, far, size, keep_first):
    """q [T, H, D], k [T, G, D] -> masked scores [H, T, T]."""
    T, H, _ = q.shape
    G = k.shape[1]
    buckets = torch.tensor([distance_bucket(n, rel.shape[0], far) for n in range(T)])
    s = torch.full((H, T, T), -math.inf, dtype=q.dtype)
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = (j <= i) & ((i - j < size) | (j < keep_first))
    b = buckets[(i - j).clamp(min=0)]
    for h in range(H):
        raw = q[:, h] @ k[:, h // (H // G)].T * scale + rel[b, h]
        s[h] = torch.where(seen, raw, s[h])
    return s


def attention_mixer(h, w, p, cfg, mix):
    """w(name) returns the tensor p + name."""
    eps = cfg["norm"]["eps"]
    H, G, D, V = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    q = rms_norm(h @ w(p + "q").T, eps, w(p + "q.norm")).view(T, H, D)
    k = rms_norm(h @ w(p + "k").T, eps, w(p + "k.norm")).view(T, G, D)
    v = (h @ w(p + "v").T).view(T, G, V)
    s = attention_scores(q, k, mix["scale"], w(p + "rel"), mix["bias_max"], mix["mask"]["size"], mix["mask"]["keep_first"])
    a = torch.softmax(s, -1)
    o = torch.stack([a[x] @ v[:, x // (H // G)] for x in range(H)], 1)
    return o.reshape(T, H * V) @ w(p + "o").T


def causal_conv_silu(x, taps):
    """x [T, C], taps [C, K]; the last column of ``taps`` belongs to the current token; zeros before the start."""
    T, C = x.shape
    K = taps.shape[1]
    pad = torch.cat([torch.zeros(K - 1, C, dtype=x.dtype), x])
    return silu(sum(pad[i:i + T] * taps[:, i] for i in range(K)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_gates(h, w, p):
    beta = torch.sigmoid(h @ w(p + "b").T)
    pre = h @ w(p + "a").T + w(p + "dt_bias")
    softplus = torch.clamp(pre, min=0) + torch.log1p(torch.exp(-pre.abs()))
    return beta, torch.exp(-torch.exp(w(p + "A_log")) * softplus)


def delta_recurrence(q, k, v, beta, g, state=None):
    """One head: q, k [T, D], v [T, V], beta, g [T] -> (o [T, V], final state [D, V])."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        S = S * g[t]
        u = beta[t] * (v[t] - k[t] @ S)
        S = S + torch.outer(k[t], u)
        out.append(q[t] @ S)
    return torch.stack(out), S


def delta_mixer(h, w, p, cfg, mix):
    H, G, D, V = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    q = causal_conv_silu(h @ w(p + "q").T, w(p + "q.conv")).view(T, G, D)
    k = causal_conv_silu(h @ w(p + "k").T, w(p + "k.conv")).view(T, G, D)
    v = causal_conv_silu(h @ w(p + "v").T, w(p + "v.conv")).view(T, H, V)
    q, k = unit(q) * D ** -0.5, unit(k)
    beta, g = delta_gates(h, w, p)
    o = torch.stack([delta_recurrence(q[:, x // (H // G)], k[:, x // (H // G)], v[:, x], beta[:, x], g[:, x])[0]
                     for x in range(H)], 1)
    o = rms_norm(o, cfg["norm"]["eps"], w(p + "norm")) * silu((h @ w(p + "g").T).view(T, H, V))
    return o.reshape(T, H * V) @ w(p + "o").T


def clamped_glu(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, -limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def feed_forward(h, w, p, mlp):
    return clamped_glu(h @ w(p + "gate").T, h @ w(p + "up").T, mlp["limit"]) @ w(p + "down").T


def forward(cfg, weights, tokens, dtype=torch.float32, keep_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    def w(name):
        return weights[name].to(dtype)

    eps = cfg["norm"]["eps"]
    x = w("embed")[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"attention": attention_mixer, "delta": delta_mixer}[layer["type"]]
        x = x + mixer(rms_norm(x, eps, w(p + "norm1")), w, p + "mix.", cfg, layer["mixer"])
        if layer["mlp"] is not None:
            x = x + feed_forward(rms_norm(x, eps, w(p + "norm2")), w, p + "mlp.", layer["mlp"])
        streams.append(x)
    logits = rms_norm(x, eps, w("final.norm")) @ w("head").T
    return (logits, streams) if keep_layers else logits
