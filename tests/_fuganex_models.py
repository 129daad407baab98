"""Small random models of the Fuganex design for the tests: configurations, weights and checkpoints."""

from __future__ import annotations

import json

import torch


def attention(heads, kv_heads, dim, vdim, window, keep_first, bias_max=40, scale=None, ff=0, limit=7.0):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                      "scale": dim ** -0.5 if scale is None else scale, "bias_max": bias_max,
                      "mask": {"size": window, "keep_first": keep_first}},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def delta(heads, kv_heads, dim, vdim, conv=4, ff=0, limit=7.0):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def config(layers, vocab=320, width=96, eps=1e-6, embed_scale=1.5):
    return {"architecture": "Fuganex", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}}


# name -> configuration. Sizes differ from layer to layer; some are odd, so that no vector path applies.
CONFIGS = {
    "mixed": config([delta(4, 2, 32, 24, 3), attention(6, 2, 24, 40, 33, 5, ff=160, limit=1.5),
                     delta(2, 2, 48, 64, 4, ff=128, limit=0.7), attention(2, 1, 64, 32, 17, 0, bias_max=90)]),
    "attention_only": config([attention(4, 4, 32, 32, 1, 3, ff=64), attention(8, 1, 16, 16, 50, 70, ff=64, scale=0.4)],
                             vocab=200, width=64),
    "delta_only": config([delta(3, 1, 40, 16, 1), delta(1, 1, 64, 128, 5, ff=96)], vocab=200, width=80, eps=1e-5),
    "odd": config([attention(3, 3, 20, 12, 40, 9, bias_max=33.5, ff=52), delta(5, 5, 12, 20, 2, ff=44)], vocab=203, width=52),
    # 16 query heads on one key head, a distance table past the tensor-core kernels' limit, windows longer than a chunk, kept
    # tokens past a chunk, a vocabulary that is no multiple of anything
    "reach": config([attention(16, 1, 16, 16, 140, 150, bias_max=4000, ff=64), delta(4, 4, 16, 32, 6),
                     attention(4, 2, 32, 64, 130, 3, bias_max=200)], vocab=331),
    "wide_head": config([attention(2, 2, 144, 160, 64, 2, ff=64), delta(2, 1, 160, 136, 4)], vocab=128, width=128),
}


def weights(cfg, seed=0, bias_rows=12, dtype=torch.bfloat16):
    """Random checkpoint tensors. Projections keep the stream's size, the distance tables and norms vary enough to show,
    and decays reach from short memories to long ones. ``bias_rows``: rows of the distance tables (per layer they differ)."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain * i ** -0.5

    def vec(n):
        return 1 + 0.3 * torch.randn(n, generator=g)

    W = cfg["width"]
    t = {"embed": torch.randn(cfg["vocab"], W, generator=g), "head": mat(cfg["vocab"], W), "final.norm": vec(W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        t[p + "norm1"] = vec(W)
        t[p + "mix.q"], t[p + "mix.k"] = mat(G * D if layer["type"] == "delta" else H * D, W), mat(G * D, W)
        t[p + "mix.o"] = mat(W, H * V)
        if layer["type"] == "attention":
            t[p + "mix.v"] = mat(G * V, W)
            t[p + "mix.q.norm"], t[p + "mix.k.norm"] = 1.5 * vec(H * D), 1.5 * vec(G * D)
            t[p + "mix.rel"] = torch.randn(bias_rows + i, H, generator=g)
        else:
            t[p + "mix.v"], t[p + "mix.g"] = mat(H * V, W), mat(H * V, W)
            t[p + "mix.b"], t[p + "mix.a"] = mat(H, W), mat(H, W)
            for x, n in (("q", G * D), ("k", G * D), ("v", H * V)):
                t[p + f"mix.{x}.conv"] = torch.randn(n, m["conv"], generator=g) * m["conv"] ** -0.5
            t[p + "mix.A_log"] = torch.rand(H, generator=g) * 3 - 2
            t[p + "mix.dt_bias"] = torch.rand(H, generator=g) * 4 - 5
            t[p + "mix.norm"] = vec(V)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            t[p + "norm2"] = vec(W)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(F, W, 2.0), mat(F, W, 2.0), mat(W, F)
    return {k: v.to(dtype) for k, v in t.items()}


def save(cfg, tensors, path):
    from safetensors.torch import save_file

    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(path / "model.safetensors"))
    return path


def load_model(cfg, tensors, path, dtype, device):
    """The framework's own way in: checkpoint folder -> configuration, registry, weights."""
    from verl_b200.models import build_model
    from verl_b200.workers.engine_workers import resolve_model_config

    mc, state = resolve_model_config({"path": str(save(cfg, tensors, path))})
    model = build_model(mc, dtype=dtype, device=device, init=False)
    model.load_state_dict(state, strict=True)
    return model


def engine(model, **kw):
    from verl_b200.rollout import NativeRolloutEngine

    args = dict(max_num_seqs=4, max_model_len=512, max_num_batched_tokens=1024, num_blocks=96, block_size=16)
    args.update(kw)
    return NativeRolloutEngine(model, **args)


def feed_portions(eng, rid, tokens, sizes, end=True):
    """All logits of one request whose tokens come in portions of the given sizes (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(k, len(sizes) - 1)], len(tokens) - at)
        last = at + n == len(tokens)
        out.append(eng.feed([(rid, tokens[at:at + n], list(range(n)))], [rid] if last and end else []).float().cpu())
        at, k = at + n, k + 1
    return torch.cat(out)


def error(got, want):
    """Largest root-mean-square difference of a row (means taken off) in units of the rows' spread."""
    got, want = got.float().cpu(), want.float()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.std(-1).mean())
