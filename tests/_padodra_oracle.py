"""Plain, slow implementation of the Padodra design on the CPU: the yardstick of ``test_padodra_*.py``.

One function per mechanism, written from the equations and sharing nothing with the package. ``weights`` maps checkpoint
tensor names to tensors, ``cfg`` is the parsed ``config.json``. Everything runs in the dtype of the weights after
``to(dtype)`` (float32 or float64).
"""

from __future__ import annotations

import math

import torch


def rms_norm(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def plain_frequencies(dims, base):
    return [base ** (-2 * i / dims) for i in range(dims // 2)]


def llama3_frequencies(dims, base, scaling):
    """Long wavelengths are slowed down by ``factor``, short ones kept, a linear blend in wavelength count between."""
    out = []
    for f in plain_frequencies(dims, base):
        turns = scaling["original"] * f / (2 * math.pi)  # full turns over the original context
        if turns > scaling["high"]:
            out.append(f)
        elif turns < scaling["low"]:
            out.append(f / scaling["factor"])
        else:
            s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
            out.append((1 - s) * f / scaling["factor"] + s * f)
    return out


def yarn_frequencies(dims, base, scaling):
    """(frequencies, factor of cos and sin): a linear ramp over the pair index from kept to slowed down."""
    def index(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(index(scaling["fast"])), 0)
    hi = min(math.ceil(index(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate(x, freqs, interleaved, factor=1.0):
    """x [T, ..., D]: the first 2 * len(freqs) dimensions turn by position * frequency; row t is position t."""
    n = len(freqs)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)
    a = a.reshape([x.shape[0]] + [1] * (x.dim() - 2) + [n])
    c, s = (torch.cos(a) * factor).to(x.dtype), (torch.sin(a) * factor).to(x.dtype)
    y = x.clone()
    iu = [2 * i for i in range(n)] if interleaved else list(range(n))
    iv = [2 * i + 1 for i in range(n)] if interleaved else list(range(n, 2 * n))
    u, v = x[..., iu], x[..., iv]
    y[..., iu] = u * c - v * s
    y[..., iv] = v * c + u * s
    return y


def chunk_mask(T, size):
    """[T, T]: query i sees key j <= i of the same chunk of ``size`` positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def causal_mask(T):
    return torch.arange(T)[None, :] <= torch.arange(T)[:, None]


def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def softmax_with_sink(s, sink=None):
    """s [..., keys]; ``sink`` joins the denominator only."""
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, torch.as_tensor(sink, dtype=s.dtype))
    e = torch.exp(s - m)
    d = e.sum(-1, keepdim=True)
    if sink is not None:
        d = d + torch.exp(torch.as_tensor(sink, dtype=s.dtype) - m)
    return e / d


def attend(q, k, v, scale, mask, cap=None, sinks=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        if cap is not None:
            s = softcap(s, cap)
        s = torch.where(mask, s, torch.full_like(s, -math.inf))
        out.append(softmax_with_sink(s, None if sinks is None else sinks[h]) @ v[:, h // (H // G)])
    return torch.stack(out, 1)


def attention_mixer(h, w, p, cfg, mix):
    eps, rot = cfg["norm"]["eps"], mix["rot"]
    H, G, D, V = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    freqs = llama3_frequencies(rot["dims"], rot["base"], rot["scaling"])
    q = rotate(rms_norm((h @ w(p + "q").T).view(T, H, D), eps, w(p + "q.norm")), freqs, True)
    k = rotate(rms_norm((h @ w(p + "k").T).view(T, G, D), eps, w(p + "k.norm")), freqs, True)
    v = (h @ w(p + "v").T).view(T, G, V)
    o = attend(q, k, v, mix["scale"], chunk_mask(T, mix["mask"]["size"]), mix["softcap"], w(p + "sink"))
    return (o.reshape(T, H * V) * sigmoid(h @ w(p + "g").T)) @ w(p + "o").T


def latent_keys_values(h, w, p, eps, mix, freqs, factor):
    """Keys [T, H, dim + rot_dim] and values [T, H, vdim] of all heads from one latent per token."""
    T, H, R = h.shape[0], mix["heads"], mix["kv_rank"]
    d = h @ w(p + "dkv").T
    c = rms_norm(d[:, :R], eps, w(p + "dkv.norm"))
    kr = rotate(d[:, R:], freqs, False, factor)
    k = (c @ w(p + "uk").T).view(T, H, mix["dim"])
    v = (c @ w(p + "uv").T).view(T, H, mix["vdim"])
    return torch.cat([k, kr[:, None].expand(T, H, mix["rot_dim"])], -1), v


def latent_mixer(h, w, p, cfg, mix):
    H, N, T = mix["heads"], mix["dim"], h.shape[0]
    freqs, factor = yarn_frequencies(mix["rot"]["dims"], mix["rot"]["base"], mix["rot"]["scaling"])
    q = (h @ w(p + "q").T).view(T, H, N + mix["rot_dim"])
    q = torch.cat([q[..., :N], rotate(q[..., N:], freqs, False, factor)], -1)
    k, v = latent_keys_values(h, w, p, cfg["norm"]["eps"], mix, freqs, factor)
    o = attend(q, k, v, mix["scale"], causal_mask(T))
    return (o.reshape(T, H * mix["vdim"]) * sigmoid(h @ w(p + "g").T)) @ w(p + "o").T


def feed_forward(h, w, p):
    return (gelu_tanh(h @ w(p + "gate").T) * (h @ w(p + "up").T)) @ w(p + "down").T


def forward(cfg, weights, tokens, dtype=torch.float32, keep_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    def w(name):
        return weights[name].to(dtype)

    eps = cfg["norm"]["eps"]
    x = w("embed")[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"attention": attention_mixer, "latent_attention": latent_mixer}[layer["type"]]
        x = x + rms_norm(mixer(x, w, p + "mix.", cfg, layer["mixer"]), eps, w(p + "norm1"))
        if layer["mlp"] is not None:
            x = x + rms_norm(feed_forward(x, w, p + "mlp."), eps, w(p + "norm2"))
        streams.append(x)
    logits = rms_norm(x, eps, w("final.norm")) @ w("head").T * cfg["logit_scale"]
    return (logits, streams) if keep_layers else logits
