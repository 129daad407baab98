"""Small random models of the Malinex design for the tests: configurations, weights and checkpoints."""

from __future__ import annotations

import torch

from _fuganex_models import engine, error, feed_portions, load_model, save  # noqa: F401  (the same for every layer-list design)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return {**d, "shared": {"ff": shared}} if shared else d


def attention(heads, kv_heads, dim, vdim, temp=(0.4, 30), scale=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def gla(heads, dim, vdim, tau=8.0, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def again(layers, j):
    """Layer j once more, with its weights."""
    return {**layers[j], "weights_of": j}


def config(layers, vocab=312, width=104, eps=1e-6, scale=0.7, positions=600):
    layers = [again(layers, x) if isinstance(x, int) else x for x in layers]
    return {"architecture": "Malinex", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "logit_scale": scale, "max_positions": positions}


# name -> configuration; a number in the list: that layer once more. Sizes differ from layer to layer; some are odd, so that no
# vector or tensor-core path applies.
CONFIGS = {
    "mixed": config([gla(3, 24, 40, 5.0, dense(160)), attention(6, 2, 24, 40, mlp=moe(5, 2, 48, 72)), 0, gla(2, 48, 16, 24.5, moe(6, 3, 40)),
                     1, 3, attention(2, 1, 64, 32, None, mlp=dense(88))]),
    "attention_only": config([attention(4, 4, 32, 32, (1.3, 1), mlp=moe(4, 4, 64, 64)), attention(8, 1, 16, 24, (-0.3, 7.5), 0.6)],
                             vocab=200, width=64, scale=1.0),
    "gla_only": config([gla(4, 32, 32, 1.0, moe(8, 1, 32, 40)), gla(1, 64, 128, 16.0), gla(5, 8, 16, 2.0, dense(72)), 1], vocab=200,
                       width=72, eps=1e-3),
    "odd": config([attention(3, 3, 20, 12, (0.7, 11), mlp=moe(3, 2, 52, 44)), gla(5, 12, 20, 3.0, moe(2, 1, 22, 18)), 0,
                   gla(3, 7, 9, 6.0, dense(37))], vocab=203, width=52, positions=301),
    # 16 query heads on one key head, the largest heads of the tensor-core kernels, values in two blocks, a wide layer used twice
    "reach": config([attention(16, 1, 16, 16, (0.2, 64), mlp=moe(12, 3, 64, 64)), gla(2, 128, 136, 12.0), attention(4, 2, 128, 128, (0.3, 50)),
                     gla(3, 72, 64, 4.0, moe(40, 5, 16, 24)), 2, 1], vocab=331),
    "wide_head": config([attention(2, 2, 144, 160, (0.5, 20), mlp=moe(4, 2, 64, 64)), gla(2, 160, 136, 7.0, dense(128))], vocab=128, width=128),
}
RANKS = (8, 5, 16, 12, 40)  # of the decays, by layer


CODES = 16


def clear_choices(cfg, t, g):
    """Routers whose choice does not hang on rounding: the first dimensions of the stream say which of ``CODES`` kinds a token is
    (no layer writes there), and a router scores the experts by kind, the chosen ones well apart from the others."""
    for n, w in t.items():
        if n == "embed":
            w[:, :CODES] = 1.8 * torch.eye(CODES)[torch.arange(w.shape[0]) % CODES]
        elif n == "pos":
            w[:, :CODES] = 0
        elif n.endswith((".norm1b", ".norm2b")):
            w[:CODES] = 0
        elif n.endswith(".norm2"):
            w[:CODES] = 1
        elif n.endswith(".router"):
            E, top = w.shape[0], cfg["layers"][int(n[1:].split(".")[0])]["mlp"]["router"]["top"]
            corr = t[n.replace("router", "correction")]
            kinds = None
            while kinds is None:
                kinds = clear_kinds(corr, E, top, g)
                if kinds is None:
                    corr.copy_((torch.rand(E, generator=g) / E).to(torch.bfloat16))
            w[:] = 0
            w[:, :CODES] = kinds.T


def clear_kinds(corr, E, top, g):
    """[CODES, E] logits whose choice is clear whatever the size of the stream, or None if none are found."""
    out = []
    corr.copy_(corr.to(torch.bfloat16))  # as it is stored
    for _ in range(CODES):
        for _ in range(200):
            z = torch.linspace(-1.2, 1.2, E)[torch.randperm(E, generator=g)]
            ranked = [(torch.softmax(a * z, -1) + corr).sort(descending=True) for a in (1.0, 1.5, 2.0, 3.0, 4.0, 5.0)]
            chosen = {tuple(sorted(s.indices[:top].tolist())) for s in ranked}
            if top == E or len(chosen) == 1 and all(float(s.values[top - 1] - s.values[top]) > 0.1 / E for s in ranked):
                out.append(z)
                break
        else:
            return None
    return torch.stack(out)


def weights(cfg, seed=0, dtype=torch.bfloat16, clear=True):
    """Random checkpoint tensors: scores that stand apart, distance biases from none to steep, decays from short memories to long
    ones. ``clear``: see :func:`clear_choices`."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain * i ** -0.5

    def vec(n, mean=1.0):
        return mean * (1 + 0.3 * torch.randn(n, generator=g))

    W = cfg["width"]
    t = {"embed": torch.randn(cfg["vocab"], W, generator=g) * 0.3, "pos": torch.randn(cfg["max_positions"], W, generator=g) * 0.2,
         "head": mat(cfg["vocab"], W), "final.norm": vec(W)}
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        p, m = f"l{i}.", layer["mixer"]
        H, D, V = m["heads"], m["dim"], m["vdim"]
        for n in (1, 2) if layer["mlp"] is not None else (1,):
            t[p + f"norm{n}"], t[p + f"norm{n}b"] = vec(W), vec(W, 0.4)
            t[p + f"rg{n}"], t[p + f"rg{n}.b"] = mat(W, W), torch.randn(W, generator=g)
        t[p + "mix.o"] = mat(W, H * V)
        if layer["type"] == "attention":
            for x, n in (("q", H * D), ("k", m["kv_heads"] * D), ("v", m["kv_heads"] * V)):
                t[p + f"mix.{x}"], t[p + f"mix.{x}.b"] = mat(n, W), 0.3 * torch.randn(n, generator=g)
                if x != "v":
                    t[p + f"mix.{x}.norm"] = vec(n, 1.5)
            t[p + "mix.r1"], t[p + "mix.r2"] = torch.rand(H, generator=g) * 1.5, torch.rand(H, generator=g) + 0.05
            t[p + "mix.r1"][0] = 0.0
            t[p + "mix.pb"] = -3.0 + torch.randn(H, generator=g)
            t[p + "mix.g"] = mat(H, W, 2.0)
        else:
            R = RANKS[i % len(RANKS)]
            for x, n in (("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V), ("a1", R)):
                t[p + f"mix.{x}"] = mat(n, W)
            t[p + "mix.a2"], t[p + "mix.a2.b"] = mat(H * D, R, 1.5), torch.rand(H * D, generator=g) * 9 - 3
            t[p + "mix.norm"] = vec(V)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            t[p + "mlp.up"], t[p + "mlp.down"] = mat(mlp["ff"], W, 2.0), mat(W, mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        t[p + "mlp.router"], t[p + "mlp.correction"] = mat(E, W, 3.0), torch.rand(E, generator=g) / E
        units = [(f"e{e}", mlp["expert"]["ff"]) for e in range(E)] + ([("shared", mlp["shared"]["ff"])] if "shared" in mlp else [])
        for x, f in units:
            t[p + f"mlp.{x}.up"], t[p + f"mlp.{x}.down"] = mat(f, W, 1.5), mat(W, f)
    if clear:
        clear_choices(cfg, t, g)
    return {k: v.to(dtype) for k, v in t.items()}
