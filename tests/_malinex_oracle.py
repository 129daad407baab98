"""Plain, slow implementation of the Malinex design on the CPU: the yardstick of ``test_malinex_*.py``.

One function per mechanism, written from the equations and sharing nothing with the package. ``weights`` maps checkpoint
tensor names to tensors, ``cfg`` is the parsed ``config.json``. Everything runs in the dtype of the weights after
``to(dtype)`` (float32 or float64).
"""

from __future__ import annotations

import math

import torch

from _padodra_oracle import causal_mask, rms_norm, sigmoid


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    """log(1 / (1 + e^-z)) without overflow."""
    return torch.minimum(z, torch.zeros_like(z)) - torch.log1p(torch.exp(-z.abs()))


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2)))


def relu2(z):
    return torch.clamp(z, min=0) ** 2


# ------------------------------------------------------------------------------------------- gated linear attention
def decays(z, tau):
    """Per key channel: sigmoid(z) to the power 1 / tau."""
    return torch.exp(log_sigmoid(z) / tau)


def linear_attention(q, k, v, a, state=None):
    """q, k, a [T, H, D], v [T, H, V]: rows of the state fade by a, then k v^T is added. ([T, H, V], state [H, D, V])."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]) if state is None else state
    out = []
    for t in range(q.shape[0]):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def gla_mixer(h, w, p, cfg, mix):
    T, H, D, V = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = (h @ w(p + "q").T).view(T, H, D) * D ** -0.5
    k = (h @ w(p + "k").T).view(T, H, D)
    v = (h @ w(p + "v").T).view(T, H, V)
    z = h @ w(p + "a1").T @ w(p + "a2").T + w(p + "a2.b")
    o, _ = linear_attention(q, k, v, decays(z, mix["tau"]).view(T, H, D))
    o = rms_norm(o, cfg["norm"]["eps"], w(p + "norm")).reshape(T, H * V)
    return (o * silu(h @ w(p + "g").T)) @ w(p + "o").T


# ------------------------------------------------------------------------------------------------ sigmoid attention
def query_temperature(positions, temp):
    """What queries are multiplied by at these positions."""
    if not temp:
        return torch.ones(len(positions), dtype=torch.float64)
    return torch.tensor([1 + temp["coef"] * math.log(math.floor((p + 1) / temp["every"]) + 1) for p in positions],
                        dtype=torch.float64)


def distance_bias(T, r1, r2):
    """[H, T, T], to be taken off: r1 ln(1 + r2 (i - j)) for j <= i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    d = (i - j).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * d)


def sigmoid_attend(q, k, v, scale, bias, shift):
    """q [T, H, D], k [T, G, D], v [T, G, V]; every visible key weighs the sigmoid of its score, whatever the others have."""
    T, H, rep = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    out = []
    for h in range(H):
        score = (q[:, h] @ k[:, h // rep].T) * scale - bias[h] + shift[h]
        weight = torch.where(causal_mask(T), sigmoid(score), torch.zeros_like(score))
        out.append(weight @ v[:, h // rep])
    return torch.stack(out, 1)


def attention_mixer(h, w, p, cfg, mix):
    T, H, G, D, V = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    eps = cfg["norm"]["eps"]
    q = rms_norm(h @ w(p + "q").T + w(p + "q.b"), eps, w(p + "q.norm"))
    k = rms_norm(h @ w(p + "k").T + w(p + "k.b"), eps, w(p + "k.norm"))
    v = h @ w(p + "v").T + w(p + "v.b")
    q = q * query_temperature(range(T), mix.get("q_temp")).to(q.dtype)[:, None]
    o = sigmoid_attend(q.view(T, H, D), k.view(T, G, D), v.view(T, G, V), mix["scale"],
                       distance_bias(T, w(p + "r1"), w(p + "r2")), w(p + "pb"))
    o = o * sigmoid(h @ w(p + "g").T)[:, :, None]
    return o.reshape(T, H * V) @ w(p + "o").T


# ---------------------------------------------------------------------------------------------------- feed-forward
def route(h, router, correction, top):
    """Chosen experts [T, top] and their weights: chosen by score plus correction, weighted by the scores' shares."""
    s = torch.softmax(h @ router.T, -1)
    idx = torch.argsort(s + correction, dim=-1, descending=True, stable=True)[:, :top]
    weight = s.gather(1, idx)
    return idx, weight / (weight.sum(-1, keepdim=True) + 1e-20)


def two_layers(x, w, p, act):
    return act(x @ w(p + "up").T) @ w(p + "down").T


def feed_forward(h, w, p, mlp):
    if mlp["kind"] == "dense":
        return two_layers(h, w, p, gelu)
    idx, weight = route(h, w(p + "router"), w(p + "correction"), mlp["router"]["top"])
    out = two_layers(h, w, p + "shared.", relu2) if mlp.get("shared") else torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if len(t):
            out[t] = out[t] + two_layers(h[t], w, p + f"e{e}.", relu2) * weight[t, k][:, None]
    return out


# ------------------------------------------------------------------------------------------------------------ model
MIXERS = {"attention": attention_mixer, "gla": gla_mixer}


def sublayer(x, w, p, n, eps, run):
    """x plus the normed, gated result of a sublayer that reads the normed x."""
    h = rms_norm(x, eps, w(f"{p}norm{n}"))
    y = run(h) * sigmoid(h @ w(f"{p}rg{n}").T + w(f"{p}rg{n}.b"))
    return x + rms_norm(y, eps, w(f"{p}norm{n}b"))


def forward(cfg, weights, tokens, dtype=torch.float32, keep_layers=False):
    """Logits [T, vocab] of one sequence (and the stream behind each layer)."""
    def w(name):
        return weights[name].to(dtype)

    eps, ids = cfg["norm"]["eps"], torch.tensor(tokens)
    x = w("embed")[ids] + w("pos")[: len(ids)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer['weights_of'] if layer.get('weights_of') is not None else i}."
        x = sublayer(x, w, p, 1, eps, lambda h: MIXERS[layer["type"]](h, w, p + "mix.", cfg, layer["mixer"]))
        if layer["mlp"] is not None:
            x = sublayer(x, w, p, 2, eps, lambda h: feed_forward(h, w, p + "mlp.", layer["mlp"]))
        streams.append(x)
    logits = rms_norm(x, eps, w("final.norm")) @ w("head").T * cfg["logit_scale"]
    return (logits, streams) if keep_layers else logits
