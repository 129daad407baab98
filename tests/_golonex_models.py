"""Small random models of the Golonex design for the tests: configurations, weights and checkpoints."""

from __future__ import annotations

import torch

from _fuganex_models import engine, error, feed_portions, load_model, save  # noqa: F401  (the same for every layer-list design)

YARN = {"factor": 5.0, "fast": 24.0, "original": 900, "slow": 1.5}


def moe(experts, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}


def attention(heads, kv_heads, dim, window, rot=None, base=3000.0, scaling=YARN, scale=None, mlp=None):
    rotary = {"dims": dim if rot is None else rot, "base": base}
    if scaling:
        rotary["scaling"] = dict(scaling)
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": rotary,
                      "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window}},
            "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, rank, q_rank, window, base=2000.0, scaling=None, scale=None, mlp=None):
    rotary = {"dims": rot_dim, "base": base}
    if scaling:
        rotary["scaling"] = dict(scaling)
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                      "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": rotary, "mask": {"size": window}},
            "mlp": mlp}


def rglru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def config(layers, vocab=304, width=96, eps=1e-6, side=16, cap=9.0):
    return {"architecture": "Golonex", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "token_side": {"dim": side}, "logit_softcap": cap}


# name -> configuration. Sizes differ from layer to layer; some are odd, so that no vector or tensor-core path applies.
CONFIGS = {
    "mixed": config([rglru(144, 3, 4, moe(5, 2, 48, 72)), attention(6, 3, 32, 37, rot=16, mlp=moe(8, 1, 64, 40)),
                     latent(4, 24, 16, 40, 48, 56, 45), rglru(96, 1, 1), latent(3, 40, 32, 16, 72, 32, 23, mlp=moe(3, 3, 40, 56)),
                     attention(4, 1, 48, 50, scaling=None, mlp=moe(7, 4, 32, 24))]),
    "attention_only": config([attention(4, 4, 32, 1, mlp=moe(4, 2, 64, 64)), attention(8, 1, 16, 300, rot=8, scale=0.6)],
                             vocab=200, width=64, side=24),
    "latent_only": config([latent(2, 16, 16, 24, 32, 24, 1), latent(5, 32, 8, 32, 136, 48, 130, scale=0.3, scaling=YARN,
                                                                   mlp=moe(6, 2, 48, 96))], vocab=200, width=80, eps=1e-3),
    "recurrent_only": config([rglru(64, 4, 2, moe(4, 1, 32, 32)), rglru(200, 1, 7), rglru(72, 9, 3, moe(40, 5, 16, 24))],
                             vocab=200, width=64, side=8),
    "odd": config([attention(3, 3, 20, 29, rot=6, mlp=moe(3, 2, 52, 44)), latent(5, 12, 6, 20, 28, 34, 31, mlp=moe(5, 1, 28, 36)),
                   rglru(60, 5, 3, moe(2, 1, 22, 18))], vocab=203, width=52, side=11),
    # 16 query heads on one key head, windows longer than a block of keys, as many heads as several groups, ranks and blocks of
    # the recurrence over several tiles, a vocabulary that is no multiple of anything
    "reach": config([attention(16, 1, 16, 141, mlp=moe(12, 3, 64, 64)), latent(36, 16, 16, 16, 200, 40, 150), rglru(272, 2, 4),
                     attention(4, 2, 128, 130, rot=80), latent(2, 128, 64, 128, 512, 192, 190, mlp=moe(4, 2, 72, 128)),
                     rglru(384, 1, 5)], vocab=331),
    "wide_head": config([attention(2, 2, 144, 64, mlp=moe(4, 2, 64, 64)), latent(2, 136, 64, 144, 96, 64, 77),
                         rglru(640, 1, 3)], vocab=128, width=128),
}


CODES = 16


def clear_choices(cfg, t, g):
    """Routers whose choice does not hang on rounding: the first dimensions of the stream say which of ``CODES`` kinds a token is
    (no layer writes there), and a router ranks the experts by kind, with scores well apart."""
    for n, w in t.items():
        if n == "embed":
            w[:, :CODES] = 1.2 * torch.eye(CODES)[torch.arange(w.shape[0]) % CODES]
        elif n.endswith((".mix.o", ".down", ".side.proj")):
            w[:CODES] = 0
        elif n == "embed.norm" or n.endswith(".norm2"):
            w[:CODES] = 1
        elif n.endswith(".router"):
            E = w.shape[0]
            w[:] = 0
            for c in range(CODES):
                w[:, c] = torch.linspace(-2.5, 2.5, E)[torch.randperm(E, generator=g)] if E > 1 else 1.0


def weights(cfg, seed=0, dtype=torch.bfloat16, clear=True):
    """Random checkpoint tensors: scores that stand apart, sinks from negligible to large, decays from short memories to long
    ones. ``clear``: see :func:`clear_choices`."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain * i ** -0.5

    def vec(n, mean=1.0):
        return mean + 0.3 * torch.randn(n, generator=g)

    W, side = cfg["width"], cfg["token_side"]["dim"]
    t = {"embed": torch.randn(cfg["vocab"], W, generator=g) * 0.3, "embed.norm": vec(W), "final.norm": vec(W),
         "side.embed": torch.randn(cfg["vocab"], side * len(cfg["layers"]), generator=g)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        t[p + "norm1"] = vec(W)
        if layer["type"] == "attention":
            H, G, D = m["heads"], m["kv_heads"], m["dim"]
            t[p + "mix.q"], t[p + "mix.k"], t[p + "mix.o"] = mat(H * D, W, 1.6), mat(G * D, W, 1.6), mat(W, H * D)
        elif layer["type"] == "latent_attention":
            H, D, V, R, Q, rot = (m[k] for k in ("heads", "dim", "vdim", "kv_rank", "q_rank", "rot_dim"))
            t[p + "mix.dq"], t[p + "mix.dq.norm"], t[p + "mix.uq"] = mat(Q, W), vec(Q), mat(H * (D + rot), Q, 2.0)
            t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = mat(R + rot, W), vec(R)
            t[p + "mix.uk"], t[p + "mix.uv"] = mat(H * D, R), mat(H * V, R)
            t[p + "mix.sink"] = 2 * torch.randn(H, generator=g)
            t[p + "mix.g"], t[p + "mix.o"] = mat(H, W, 2.0), mat(W, H * V)
        else:
            C, B, taps = m["width"], m["blocks"], m["conv"]
            n = C // B
            for x in ("y", "x"):
                t[p + f"mix.{x}"], t[p + f"mix.{x}.b"] = mat(C, W), 0.5 * torch.randn(C, generator=g)
            t[p + "mix.conv"] = torch.randn(C, taps, generator=g) * taps ** -0.5
            t[p + "mix.conv.b"] = 0.3 * torch.randn(C, generator=g)
            for x in ("ra", "ri"):
                t[p + f"mix.{x}"] = torch.randn(B, n, n, generator=g) * 2 * n ** -0.5
                t[p + f"mix.{x}.b"] = torch.randn(B, n, generator=g)
            t[p + "mix.lam"] = torch.rand(C, generator=g) * 7 - 6
            t[p + "mix.o"] = mat(W, C)
        if layer["mlp"] is not None:
            E, F = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            t[p + "norm2"] = vec(W)
            t[p + "mlp.router"] = mat(E, W, 3.0)
            for x, f in [(f"e{e}", F) for e in range(E)] + [("shared", layer["mlp"]["shared"]["ff"])]:
                t[p + f"mlp.{x}.gate"], t[p + f"mlp.{x}.up"], t[p + f"mlp.{x}.down"] = mat(f, W, 2.0), mat(f, W, 2.0), mat(W, f)
            t[p + "mlp.shared.sg"] = mat(1, W, 2.0)
        t[p + "side.gate"], t[p + "side.proj"], t[p + "side.norm"] = mat(side, W), mat(W, side), vec(W, 0.5)
    if clear:
        clear_choices(cfg, t, g)
    return {k: v.to(dtype) for k, v in t.items()}
