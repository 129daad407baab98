"""Small random models of the Padodra design for the tests: configurations, weights and checkpoints."""

from __future__ import annotations

import torch

from _fuganex_models import engine, error, feed_portions, load_model, save  # noqa: F401  (the same for every layer-list design)

LLAMA3 = {"factor": 6.0, "high": 5.0, "low": 1.5, "original": 700}
YARN = {"factor": 5.0, "fast": 24.0, "original": 900, "slow": 1.5}


def attention(heads, kv_heads, dim, vdim, chunk, rot=None, base=3000.0, scaling=LLAMA3, softcap=20.0, scale=None, ff=0):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                      "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap, "mask": {"size": chunk},
                      "rot": {"dims": dim if rot is None else rot, "base": base, "scaling": dict(scaling)}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot_dim, vdim, rank, base=2000.0, scaling=YARN, scale=None, ff=0):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                      "scale": (dim + rot_dim) ** -0.5 if scale is None else scale,
                      "rot": {"dims": rot_dim, "base": base, "scaling": dict(scaling)}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, vocab=304, width=96, eps=1e-6, embed_scale=3.0, logit_scale=0.7):
    return {"architecture": "Padodra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "logit_scale": logit_scale}


# name -> configuration. Sizes differ from layer to layer; some are odd, so that no vector or tensor-core path applies.
CONFIGS = {
    "mixed": config([latent(4, 24, 16, 40, 48), attention(6, 3, 32, 24, 37, rot=16, ff=160),
                     latent(3, 40, 32, 16, 72, ff=128), attention(4, 1, 48, 64, 50)]),
    "attention_only": config([attention(4, 4, 32, 32, 1, ff=64), attention(8, 1, 16, 16, 300, softcap=1.5, ff=64, scale=0.6)],
                             vocab=200, width=64),
    "latent_only": config([latent(2, 16, 16, 24, 32), latent(5, 32, 8, 32, 136, ff=96, scale=0.3)], vocab=200, width=80, eps=1e-3),
    "odd": config([attention(3, 3, 20, 12, 29, rot=6, ff=52), latent(5, 12, 6, 20, 28, ff=44)], vocab=203, width=52),
    # 16 query heads on one key head, chunks longer than a block of keys, as many heads as several groups, ranks over several
    # blocks, a vocabulary that is no multiple of anything
    "reach": config([attention(16, 1, 16, 16, 141, ff=64), latent(36, 16, 16, 16, 200), attention(4, 2, 128, 64, 130, rot=80),
                     latent(2, 128, 64, 128, 512, ff=72)], vocab=331),
    "wide_head": config([attention(2, 2, 144, 160, 64, ff=64), latent(2, 136, 64, 144, 96)], vocab=128, width=128),
}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random checkpoint tensors: query and key norms above one make the scores stand apart, sinks from negligible to large."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain * i ** -0.5

    def vec(n, mean=1.0):
        return mean + 0.3 * torch.randn(n, generator=g)

    W = cfg["width"]
    # sublayers read the stream as it is: the projections undo its scale
    gain = 1 / cfg["embedding"]["scale"]
    t = {"embed": torch.randn(cfg["vocab"], W, generator=g), "head": mat(cfg["vocab"], W), "final.norm": vec(W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, D, V = m["heads"], m["dim"], m["vdim"]
        t[p + "norm1"] = vec(W)
        if layer["type"] == "attention":
            G = m["kv_heads"]
            t[p + "mix.q"], t[p + "mix.k"], t[p + "mix.v"] = mat(H * D, W, gain), mat(G * D, W, gain), mat(G * V, W, gain)
            t[p + "mix.q.norm"], t[p + "mix.k.norm"] = vec(D, 1.6), vec(D, 1.6)
            t[p + "mix.sink"] = 2 * torch.randn(H, generator=g)
        else:
            R, rot = m["kv_rank"], m["rot_dim"]
            t[p + "mix.q"], t[p + "mix.dkv"] = mat(H * (D + rot), W, 2 * gain), mat(R + rot, W, gain)
            t[p + "mix.dkv.norm"] = vec(R)
            t[p + "mix.uk"], t[p + "mix.uv"] = mat(H * D, R), mat(H * V, R)
        t[p + "mix.g"], t[p + "mix.o"] = mat(H * V, W, gain), mat(W, H * V)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            t[p + "norm2"] = vec(W)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(F, W, gain), mat(F, W, gain), mat(W, F)
    return {k: v.to(dtype) for k, v in t.items()}
