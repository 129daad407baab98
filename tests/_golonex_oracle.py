"""Plain, slow implementation of the Golonex design on the CPU: the yardstick of ``test_golonex_*.py``.

One function per mechanism, written from the equations and sharing nothing with the package. ``weights`` maps checkpoint
tensor names to tensors, ``cfg`` is the parsed ``config.json``. Everything runs in the dtype of the weights after
``to(dtype)`` (float32 or float64).
"""

from __future__ import annotations

import torch

from _padodra_oracle import attend, causal_mask, gelu_tanh, plain_frequencies, rms_norm, rotate, sigmoid, yarn_frequencies  # noqa: F401


def window_mask(T, size):
    """[T, T]: query i sees the keys i - size + 1 .. i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    """log(1 + e^z) without overflow."""
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(x, kernel, bias):
    """x [T, C], kernel [C, taps]: column j meets the input taps - 1 - j tokens back, if there is one."""
    T, taps = x.shape[0], kernel.shape[1]
    y = torch.zeros_like(x) + bias
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] = y[back:] + x[: T - back] * kernel[:, j]
    return y


def block_linear(x, blocks, bias):
    """x [T, C] in equal parts, blocks [n, C / n, C / n] (out, in), bias [n, C / n]."""
    n, size, _ = blocks.shape
    return torch.cat([x[:, b * size : (b + 1) * size] @ blocks[b].T + bias[b] for b in range(n)], -1)


def lru_gates(u, r, i, lam):
    """Decay and input of the recurrence per channel."""
    log_a = -8 * r * softplus(lam)
    a = torch.exp(log_a)
    return a, torch.sqrt(1 - a * a) * i * u


def linear_scan(a, b, state=None):
    """S_t = a_t S_(t-1) + b_t, row by row."""
    S, out = torch.zeros_like(a[0]) if state is None else state, []
    for t in range(a.shape[0]):
        S = a[t] * S + b[t]
        out.append(S)
    return torch.stack(out)


def rglru_mixer(h, w, p, cfg, mix):
    y = gelu_tanh(h @ w(p + "y").T + w(p + "y.b"))
    u = causal_conv(h @ w(p + "x").T + w(p + "x.b"), w(p + "conv"), w(p + "conv.b"))
    r, i = (sigmoid(block_linear(u, w(p + g), w(p + g + ".b"))) for g in ("ra", "ri"))
    S = linear_scan(*lru_gates(u, r, i, w(p + "lam")))
    return (S * y) @ w(p + "o").T


def rotation(rot):
    if rot.get("scaling"):
        return yarn_frequencies(rot["dims"], rot["base"], rot["scaling"])
    return plain_frequencies(rot["dims"], rot["base"]), 1.0


def attention_mixer(h, w, p, cfg, mix):
    """Grouped attention whose values are the unrotated keys."""
    H, G, D = mix["heads"], mix["kv_heads"], mix["dim"]
    T = h.shape[0]
    freqs, factor = rotation(mix["rot"])
    q = rotate((h @ w(p + "q").T).view(T, H, D), freqs, True, factor)
    v = (h @ w(p + "k").T).view(T, G, D)
    o = attend(q, rotate(v, freqs, True, factor), v, mix["scale"], window_mask(T, mix["mask"]["size"]))
    return o.reshape(T, H * D) @ w(p + "o").T


def latent_queries(h, w, p, eps, mix, freqs, factor):
    """[T, heads, dim + rot_dim] out of a normed latent; the last rot_dim turn."""
    N = mix["dim"]
    q = rms_norm(h @ w(p + "dq").T, eps, w(p + "dq.norm")) @ w(p + "uq").T
    q = q.view(h.shape[0], mix["heads"], N + mix["rot_dim"])
    return torch.cat([q[..., :N], rotate(q[..., N:], freqs, True, factor)], -1)


def latent_keys_values(h, w, p, eps, mix, freqs, factor):
    """Keys [T, H, dim + rot_dim] and values [T, H, vdim] of all heads from one latent per token."""
    T, H, R = h.shape[0], mix["heads"], mix["kv_rank"]
    d = h @ w(p + "dkv").T
    c = rms_norm(d[:, :R], eps, w(p + "dkv.norm"))
    kr = rotate(d[:, R:], freqs, True, factor)
    k = (c @ w(p + "uk").T).view(T, H, mix["dim"])
    v = (c @ w(p + "uv").T).view(T, H, mix["vdim"])
    return torch.cat([k, kr[:, None].expand(T, H, mix["rot_dim"])], -1), v


def latent_mixer(h, w, p, cfg, mix):
    T, eps = h.shape[0], cfg["norm"]["eps"]
    turn = rotation(mix["rot"])
    q = latent_queries(h, w, p, eps, mix, *turn)
    k, v = latent_keys_values(h, w, p, eps, mix, *turn)
    o = attend(q, k, v, mix["scale"], window_mask(T, mix["mask"]["size"]), None, w(p + "sink"))
    return (o * sigmoid(h @ w(p + "g").T)[:, :, None]).reshape(T, -1) @ w(p + "o").T


def glu(x, w, p, scale=None):
    x = x if scale is None else x * scale
    return (silu(x @ w(p + "gate").T) * (x @ w(p + "up").T)) @ w(p + "down").T


def route(h, router, top):
    """Chosen experts [T, top] and their weights: the sigmoid scores as they are."""
    s = sigmoid(h @ router.T)
    idx = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return idx, s.gather(1, idx)


def feed_forward(h, w, p, mlp):
    """Routed experts, each on its input times the weight, and the gated shared expert."""
    idx, weight = route(h, w(p + "router"), mlp["router"]["top"])
    out = glu(h, w, p + "shared.") * sigmoid(h @ w(p + "shared.sg").T)
    for e in range(mlp["router"]["experts"]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if len(t):
            out[t] = out[t] + glu(h[t], w, p + f"e{e}.", weight[t, k][:, None])
    return out


def side_input(x, w, i, tokens, cfg):
    """What layer i adds to the stream out of its part of the token's side embedding."""
    n = cfg["token_side"]["dim"]
    e = w("side.embed")[tokens][:, i * n : (i + 1) * n]
    p = f"l{i}.side."
    y = (gelu_tanh(x @ w(p + "gate").T) * e) @ w(p + "proj").T
    return rms_norm(y, cfg["norm"]["eps"], w(p + "norm"))


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer, "rglru": rglru_mixer}


def forward(cfg, weights, tokens, dtype=torch.float32, keep_layers=False):
    """Logits [T, vocab] of one sequence (and the stream behind each layer)."""
    def w(name):
        return weights[name].to(dtype)

    eps, ids = cfg["norm"]["eps"], torch.tensor(tokens)
    x = rms_norm(w("embed")[ids], eps, w("embed.norm"))
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](rms_norm(x, eps, w(p + "norm1")), w, p + "mix.", cfg, layer["mixer"])
        if layer["mlp"] is not None:
            x = x + feed_forward(rms_norm(x, eps, w(p + "norm2")), w, p + "mlp.", layer["mlp"])
        x = x + side_input(x, w, i, ids, cfg)
        streams.append(x)
    cap = cfg["logit_softcap"]
    logits = cap * torch.tanh(rms_norm(x, eps, w("final.norm")) @ w("embed").T / cap)
    return (logits, streams) if keep_layers else logits
