"""Serving throughput of a layer-list model beside a homogeneous model of equal size: prefill and decode through the
rollout engine (random weights), and every kernel of the layer beside its counterpart.

    python bench.py --serving fuganex-8b [--serving-vs llama-3-8b] [--serving-layers 6] [--serving-kernels]

All times are CUDA events after warm-up on inputs larger than L2 (or rotated over enough copies). Rooflines: bytes over
the measured copy bandwidth, flops over the measured bf16 matrix throughput (``MEASURED_PEAKS.json``).
"""

from __future__ import annotations

import json
import os
from pathlib import Path

import torch

from .. import ops
from ..models import build_model, preset
from ..models.layer_specs import PLAIN_ACTS, MoeSpec
from ..ops import _lib
from ..ops import moe as moe_ops
from .engine import NativeRolloutEngine


def _peaks() -> tuple[float, float, str]:
    p = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if p.exists():
        d = json.loads(p.read_text())
        return d["hbm_gbs"], d["bf16_tflops"], "measured"
    return 6650.0, 1590.0, "fallback"


def time_us(fn, iters: int = 10, warmup: int = 3) -> float:
    """Microseconds per call: the calls are captured into one CUDA graph, so host time is not measured."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for _ in range(iters):
            fn()
    g.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    g.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters * 1e3


def model_config(name: str, layers: int):
    """The preset with ``layers`` layers (layer-list models: their first ``layers`` layers)."""
    full = preset(name)
    if full.is_layer_list:
        return preset(name, layer_specs=full.layer_specs[:layers])
    return preset(name, num_hidden_layers=layers)


def bench_model(name: str, layers: int, prefills: list[tuple[int, int]], decodes: list[tuple[int, int]], iters: int) -> dict:
    """Prefill of ``(prompts, length)`` and decode steps of ``(sequences, context)``: one engine per point."""
    dev = torch.device("cuda")
    cfg = model_config(name, layers)
    model = build_model(cfg, dtype=torch.bfloat16, device=dev)
    out = {"model": name, "layers": layers, "parameters_1e9": round(cfg.num_parameters() / 1e9, 3), "prefill": [], "decode": []}
    gen = torch.Generator().manual_seed(0)
    for B, n in prefills:
        eng = NativeRolloutEngine(model, max_num_seqs=B, max_model_len=n + 16, max_num_batched_tokens=B * n,
                                  num_blocks=B * (n // 16 + 2), enable_prefix_caching=False)
        for i in range(B):
            eng.add_request(str(i), torch.randint(100, cfg.vocab_size - 100, (n,), generator=gen).tolist(), {"max_tokens": 4})
        k, _ = eng.sched.step()
        assert k == B
        lo = [i * n for i in range(B)]

        def prefill():  # same pages, same states (they restart at position 0): the call repeats exactly
            eng._prefill_forward(list(range(B)), lo)

        for _ in range(3):
            prefill()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(iters):
            prefill()
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / iters
        out["prefill"].append({"prompts": B, "len": n, "ms": round(ms, 3), "tokens_per_s": round(B * n / ms * 1e3)})
        eng.abort_all_requests()
        eng.sleep()
        del eng
    for B, ctx in decodes:
        eng = NativeRolloutEngine(model, max_num_seqs=B, max_model_len=ctx + 16, max_num_batched_tokens=8192,
                                  num_blocks=B * (ctx // 16 + 2), enable_prefix_caching=False)
        st, graph, _ = eng._get_graph(B)
        per = (ctx + 15) // 16
        # every row at context `ctx` on pages spread over the cache; not alive, so that replays do not advance
        st["bt"][:, :per] = torch.randperm(B * per, device=dev).view(B, per).int()
        st["lens"].fill_(ctx)
        st["pos"].fill_(ctx - 1)
        st["alive"].zero_()
        st["slots"].fill_(-1)
        if cfg.is_layer_list:
            st["state"].copy_(torch.arange(B, dtype=torch.int32))
        for _ in range(3):
            graph.replay()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(5 * iters):
            graph.replay()
        e1.record()
        torch.cuda.synchronize()
        us = e0.elapsed_time(e1) / (5 * iters) * 1e3
        out["decode"].append({"sequences": B, "ctx": ctx, "us_per_step": round(us, 1), "tokens_per_s": round(B / us * 1e6)})
        eng.sleep()
        del eng
    return out


def _paged(B: int, n: int, bs: int, heads: int, dim: int):
    per = (n + bs - 1) // bs
    kc = torch.randn(B * per, heads, bs, dim, device="cuda", dtype=torch.bfloat16)
    vc = torch.randn_like(kc)
    bt = torch.randperm(B * per, device="cuda").view(B, per).int()
    return kc, vc, bt


@torch.no_grad()
def bench_kernels(name: str, vs: str, B: int, n: int, DB: int, ctx: int) -> list[dict]:
    """Kernel times of the layer-list model and of its counterparts: prefill of B x n tokens, decode of DB sequences."""
    bw, tf, _ = _peaks()
    cfg, ref = preset(name), preset(vs)
    mixers = {s.kind: s.mixer for s in reversed(cfg.layer_specs)}
    glu = next(s.mlp for s in cfg.layer_specs if s.mlp is not None)
    H, T, bf = cfg.hidden_size, B * n, torch.bfloat16
    r = lambda *s: torch.randn(*s, device="cuda", dtype=bf)  # noqa: E731
    rows = []

    def add(kernel, us, nbytes=0.0, flops=0.0):
        ideal = max(nbytes / bw / 1e3, flops / tf / 1e6)
        rows.append({"kernel": kernel, "us": round(us, 1), "roofline_us": round(ideal, 1), "frac": round(ideal / us, 3)})

    # norm with residual: fp32 stream against the bf16 stream of the homogeneous model
    x, res32, res16, w = r(T, H), torch.randn(T, H, device="cuda"), r(T, H), r(H)
    if cfg.design.norm == "both":
        g = r(T, H) if cfg.design.residual_gate else None
        add("rmsnorm_add with " + ("gate and " if g is not None else "") + "next norm (fp32 residual)", time_us(
            lambda: ops.rmsnorm_add(x, res32, w, 1e-5, final_weight=w, gate=g)), T * H * (14 if g is not None else 12))
    elif cfg.design.norm == "post":
        add("rmsnorm_add (fp32 residual)", time_us(lambda: ops.rmsnorm_add(x, res32, w, 1e-5)), T * H * 12)
    else:
        add("add_rmsnorm (fp32 residual)", time_us(lambda: ops.add_rmsnorm(x, res32, w, 1e-5)), T * H * 12)
    add("  vs rmsnorm (bf16 residual)", time_us(lambda: ops.rmsnorm(x, w, 1e-5, res16)), T * H * 8)
    routed = glu if isinstance(glu, MoeSpec) else None
    ff = routed.shared_ff if routed else glu.ff
    gu = r(T, 2 * ff)
    if glu.act in PLAIN_ACTS:
        add(f"activation ({glu.act}, {ff})", time_us(lambda: ops.activation(gu, ff, glu.act)), T * ff * 4)
    elif glu.act == "silu":
        add(f"silu_glu ({ff})", time_us(lambda: ops.silu_glu(gu, ff)), T * ff * 6)
    elif glu.act == "gelu_tanh":
        add("gelu_tanh_glu", time_us(lambda: ops.gelu_tanh_glu(gu, glu.ff)), T * glu.ff * 6)
    else:
        add("clamped_glu", time_us(lambda: ops.clamped_glu(gu, glu.ff, glu.limit, glu.alpha)), T * glu.ff * 6)
    add("  vs swiglu", time_us(lambda: ops.swiglu(gu)), T * ff * 6)
    del gu
    if cfg.side_dim:
        _bench_side(add, r, cfg, T)
    routed = routed or next((s.mlp for s in cfg.layer_specs if isinstance(s.mlp, MoeSpec)), None)
    if routed:
        _bench_moe(add, r, routed, H, T, f"prefill {T}")
        _bench_moe(add, r, routed, H, DB, f"decode {DB}")
    if "rglru" in mixers:
        _bench_lru(add, r, mixers["rglru"], B, n, DB, ctx)
    if "attention" in mixers:
        _bench_attention(add, r, mixers["attention"], ref, B, n, DB, ctx)
    if "latent_attention" in mixers:
        _bench_latent(add, r, mixers["latent_attention"], B, n, DB, ctx)
    if "delta" in mixers:
        _bench_delta(add, r, mixers["delta"], B, n, DB, ctx)
    if "gla" in mixers:
        _bench_gla(add, r, mixers["gla"], B, n, DB, ctx)
    return rows


def _slots(bt, B: int, n: int):
    return (bt.long()[:, :, None] * 16 + torch.arange(16, device="cuda")).view(B, -1)[:, :n].reshape(-1).contiguous()


def _bench_attention(add, r, att, ref, B: int, n: int, DB: int, ctx: int) -> None:
    T, hq, hk, d = B * n, att.heads, att.kv_heads, att.dim
    # query / key norm (and rotation) with the cache write against RoPE + cache write
    kc, vc, bt = _paged(B, n, 16, hk, d)
    slots = _slots(bt, B, n)
    qkv, (nqw, nkw) = r(T, att.q_size + 2 * att.k_size), att.norm_sizes
    qw, kw = r(nqw), r(nkw)
    nb = T * (2 * att.q_size + 4 * att.k_size) * 2
    pos = torch.arange(n, device="cuda").repeat(B)
    if att.rotary is not None:
        freqs = torch.tensor(att.rotary.frequencies(), device="cuda")
        if not att.qk_norm:
            qw = kw = None
        what = "no norm, values are the keys" if att.key_values else "norm per head"
        add(f"head_norm_rope_kv_write ({what})", time_us(lambda: ops.head_norm_rope_kv_write(
            qkv, qw, kw, freqs, pos, slots, kc, vc, hq, 1e-5, interleaved=att.rotary.interleaved, key_values=att.key_values)),
            nb - (T * att.k_size * 2 if att.key_values else 0))
    else:
        add("qk_norm_kv_write" + (" with query temperature" if att.q_temp else ""), time_us(lambda: ops.qk_norm_kv_write(
            qkv, qw, kw, slots, kc, vc, hq, 1e-5, q_temp=att.q_temp, positions=pos)), nb)
    cos, sin = ops.rope_tables(ref.head_dim, n, 1e6, "cuda")

    def rope_write():
        y = ops.rope_qkv(qkv, pos, cos, sin, hq, hk, d)
        ops.kv_cache_write(y[:, att.q_size : att.q_size + att.k_size].view(T, hk, d),
                           y[:, att.q_size + att.k_size :].view(T, hk, d), slots, kc, vc)

    add("  vs rope + kv_cache_write", time_us(rope_write), nb)
    # prefill attention
    qkv.normal_()
    q = qkv[:, : att.q_size].view(T, hq, d)
    cu = torch.arange(B + 1, device="cuda", dtype=torch.int32) * n
    lens = torch.full((B,), n, device="cuda", dtype=torch.int32)
    i = torch.arange(n, dtype=torch.float64)
    kw_, what = {"scale": att.scale}, []
    if att.chunk:
        pairs = float((i % att.chunk + 1).sum())
        kw_["chunk"] = att.chunk
        what.append(f"chunk {att.chunk}")
    elif att.window:
        pairs = float((torch.minimum(i + 1, torch.full_like(i, att.window) + torch.minimum(
            torch.full_like(i, att.keep_first), (i + 1 - att.window).clamp(min=0)))).sum())
        kw_ |= {"window": att.window, "keep_first": att.keep_first}
        what.append(f"window {att.window}")
    else:
        pairs = float((i + 1).sum())
    if att.bias_max:
        kw_["bias"] = torch.randn(hq, int(att.bias_max) + 1, device="cuda")
        what.append("bias")
    if att.softcap:
        kw_["softcap"] = att.softcap
        what.append("softcap")
    if att.sink:
        kw_["sink"] = torch.randn(hq, device="cuda")
        what.append("sink")
    if att.weighting == "sigmoid":
        kw_["shift"] = torch.full((hq,), -4.0, device="cuda")
        what.append("sigmoid")
    if att.log_bias:
        kw_["log_bias"] = (torch.rand(hq, device="cuda"), torch.rand(hq, device="cuda"))
        what.append("log bias")
    gate = r(max(T, DB), att.gate_size) if att.gate else None
    if att.gate:
        what.append("gate" if att.gate == "element" else f"gate per {att.gate}")
    what = ", ".join(what)
    nbytes = T * ((2 * hq + 2 * hk) * d + att.gate_size) * 2
    add(f"paged_flash ({what})", time_us(lambda: ops.paged_attention(
        q, kc, vc, bt, cu, lens, n, **kw_, gate=gate[:T] if att.gate else None)), nbytes, 4 * pairs * B * hq * d)
    add("paged_flash (full causal, plain)", time_us(
        lambda: ops.paged_attention(q, kc, vc, bt, cu, lens, n, scale=att.scale)),
        T * (2 * hq + 2 * hk) * d * 2, 2.0 * n * (n + 1) * B * hq * d)
    k = qkv[:, att.q_size : att.q_size + att.k_size].view(T, hk, d)
    v = qkv[:, att.q_size + att.k_size :].view(T, hk, d)
    add("  vs flash_fwd (full causal)", time_us(lambda: ops.attention_varlen(q, k, v, cu, n)),
        T * (2 * hq + 2 * hk) * d * 2, 2.0 * n * (n + 1) * B * hq * d)
    # decode attention
    kc, vc, bt = _paged(DB, ctx, 16, hk, d)
    q1, cu1 = r(DB, hq, d), torch.arange(DB + 1, device="cuda", dtype=torch.int32)
    lens = torch.full((DB,), ctx, device="cuda", dtype=torch.int32)
    seen = (ctx - 1) % att.chunk + 1 if att.chunk else min(ctx, att.window + att.keep_first) if att.window else ctx
    add(f"paged_decode_window ({what}: {seen} keys)", time_us(lambda: ops.paged_attention(
        q1, kc, vc, bt, cu1, lens, 1, max_ctx=ctx, **kw_, gate=gate[:DB] if att.gate else None)), DB * seen * hk * d * 4)
    splits, work = ops.decode_workspace(DB, hq, hk, d, ctx, "cuda")
    add("  vs paged_decode_tc (full context)", time_us(
        lambda: ops.paged_decode_attention(q1, kc, vc, bt, lens, num_splits=splits, work=work)), DB * ctx * hk * d * 4)


def _seen(n: int, window: int) -> float:
    """Pairs of a query and a key that it sees, for one prompt."""
    i = torch.arange(1, n + 1, dtype=torch.float64)
    return float((i.clamp(max=window) if window else i).sum())


def _bench_latent(add, r, m, B: int, n: int, DB: int, ctx: int) -> None:
    T, h, D, width = B * n, m.heads, m.dim + m.rot_dim, ops.latent_width(m.latent_size)
    per = (n + 15) // 16
    pages, bt = r(B * per, 16, width), torch.randperm(B * per, device="cuda").view(B, per).int()
    proj, nw, qw = r(T, (m.proj_size + 7) // 8 * 8), r(m.kv_rank), r(m.q_rank) if m.q_rank else None
    freqs, pos, slots = torch.tensor(m.rotary.frequencies(), device="cuda"), torch.arange(n, device="cuda").repeat(B), _slots(bt, B, n)
    q = r(T, m.q_size) if m.q_rank else proj
    lens = torch.full((B,), n, device="cuda", dtype=torch.int32)
    rot = dict(interleaved=m.rotary.interleaved)
    add("latent_rope_write" + (" (with the norm of the queries' latent)" if m.q_rank else ""), time_us(lambda: ops.latent_rope_write(
        proj, nw, freqs, pos, slots, pages, 0 if m.q_rank else h, m.dim, m.rot_dim, m.kv_rank, 1e-5, q_rank=m.q_rank, q_norm_w=qw,
        **rot)), T * 4 * ((m.q_rank or h * m.rot_dim) + m.latent_size))
    if m.q_rank:
        add("rotate_tails (queries)", time_us(lambda: ops.rotate_tails(q, freqs, pos, h, m.dim, m.rot_dim, **rot)),
            T * 4 * h * m.rot_dim)
    proj.normal_()
    q.normal_()
    q, gate = q[:, : m.q_size].view(T, h, D), proj[:, m.q_in + m.latent_size : m.proj_size] if m.gate else None
    sink = torch.randn(h, device="cuda") if m.sink else None
    kw = dict(scale=m.scale, window=m.window, sink=sink)
    what = ", ".join([f"window {m.window}" if m.window else "full causal"] + ["sink"] * m.sink
                     + [f"gate per {m.gate}"] * (m.gate is not None))
    cu = torch.arange(B + 1, device="cuda", dtype=torch.int32) * n
    up = r(m.up_size, m.kv_rank) * m.kv_rank ** -0.5
    add("latent_gather", time_us(lambda: ops.latent_gather(pages, bt, cu, T, lens)), T * width * 4)
    rows = ops.latent_gather(pages, bt, cu, T)
    add("up projection of the latents (gemm)", time_us(lambda: ops.gemm(rows[:, : m.kv_rank], up)),
        2 * (T * (m.kv_rank + m.up_size) + m.up_size * m.kv_rank), 2.0 * T * m.up_size * m.kv_rank)
    kv, out = ops.gemm(rows[:, : m.kv_rank], up), r(T, m.out_size)
    nbytes = 2 * T * (h * (D + m.dim + 2 * m.vdim) + m.rot_dim + m.gate_size)
    flops = 2.0 * _seen(n, m.window) * B * h * (D + m.vdim)
    add(f"latent_flash ({what})", time_us(lambda: ops.latent_prefill(
        q, rows[:, m.kv_rank : m.latent_size], kv, cu, cu, n, m.dim, m.vdim, gate=gate, out=out, **kw)), nbytes, flops)
    if m.window or m.sink:
        add("  vs latent_flash (full causal, plain)", time_us(lambda: ops.latent_prefill(
            q, rows[:, m.kv_rank : m.latent_size], kv, cu, cu, n, m.dim, m.vdim, scale=m.scale, gate=None, out=out)), nbytes,
            2.0 * _seen(n, 0) * B * h * (D + m.vdim))
    per = (ctx + 15) // 16
    pages, bt = r(DB * per, 16, width), torch.randperm(DB * per, device="cuda").view(DB, per).int()
    lens, cu1 = torch.full((DB,), ctx, device="cuda", dtype=torch.int32), torch.arange(DB + 1, device="cuda", dtype=torch.int32)
    uk, uv = up[: h * m.dim].view(h, m.dim, m.kv_rank), up[h * m.dim :].view(h, m.vdim, m.kv_rank)
    # the weights of the per-head products rotate, so that they come from memory
    uks, uvs = [uk.clone() for _ in range(40)], [uv.clone() for _ in range(40)]
    turn = [0]

    def at(ws):
        turn[0] += 1
        return ws[turn[0] % 40]

    add("latent_queries (decode)", time_us(lambda: ops.latent_queries(q[:DB], at(uks)), iters=40),
        2 * (h * m.dim * m.kv_rank + DB * h * (D + width)), 2.0 * DB * h * m.dim * m.kv_rank)
    qa = ops.latent_queries(q[:DB], uk)
    seen = min(ctx, m.window) if m.window else ctx
    decode = lambda **k: ops.latent_attention(qa, pages, bt, cu1, lens, m.kv_rank, max_ctx=ctx, **k)  # noqa: E731

    def cost(keys):
        return 2 * DB * (keys * m.latent_size + h * (width + m.kv_rank)), 2.0 * DB * keys * h * (m.latent_size + m.kv_rank)

    add(f"latent_decode ({what}: {seen} keys)", time_us(lambda: decode(**kw)), *cost(seen))
    if m.window or m.sink:
        add("  vs latent_decode (full context)", time_us(lambda: decode(scale=m.scale)), *cost(ctx))
    lat = decode(**kw)
    add("latent_values (decode, gate)", time_us(lambda: ops.latent_values(
        lat, at(uvs), None if gate is None else gate[:DB], out[:DB]), iters=40),
        2 * (h * m.vdim * m.kv_rank + DB * (h * (m.kv_rank + m.vdim) + m.gate_size)), 2.0 * DB * h * m.vdim * m.kv_rank)
    x, ws = r(DB, m.kv_rank), [uv.reshape(-1, m.kv_rank).clone() for _ in range(40)]
    add("  vs gemm with a weight of that size", time_us(lambda: ops.gemm(x, at(ws)), iters=40),
        2 * (h * m.vdim * m.kv_rank + DB * (m.kv_rank + h * m.vdim)), 2.0 * DB * h * m.vdim * m.kv_rank)


def _bench_side(add, r, cfg, T: int) -> None:
    H, d, L = cfg.hidden_size, cfg.side_dim, 6
    table, ids, g = r(cfg.vocab_size, L * d), torch.randint(cfg.vocab_size, (T,), device="cuda"), r(T, d)
    x, y, w, res = r(T, H), r(T, H), r(H), torch.randn(T, H, device="cuda")
    wg, wp = r(d, H) * 0.02, r(H, d) * 0.02
    add("side gate (gemm)", time_us(lambda: ops.gemm(x, wg)), 2 * (T * (H + d) + H * d), 2.0 * T * H * d)
    add("gelu_rows", time_us(lambda: ops.gelu_rows(g, ids, table, d, d)), 6 * T * d)
    add("side output (gemm)", time_us(lambda: ops.gemm(g, wp)), 2 * (T * (H + d) + H * d), 2.0 * T * H * d)
    add("rmsnorm_add with the next norm (fp32 residual)", time_us(lambda: ops.rmsnorm_add(y, res, w, 1e-5, final_weight=w)), T * H * 12)


def _bench_moe(add, r, m, H: int, T: int, tag: str) -> None:
    E, top, ff = m.experts, m.top, m.ff
    x, logits, res, w = r(T, H), torch.randn(T, (m.router_rows + 7) // 8 * 8, device="cuda"), torch.randn(T, H, device="cuda"), r(H)
    counters = torch.zeros(E + 1, dtype=torch.int32, device="cuda")
    wr = r(logits.shape[1], H) * 0.02
    copies = 1 if T > 2048 else 8  # decode: the weights rotate, so that they come from memory
    first = 2 * ff if m.gated else ff
    gus, downs = [r(E, first, H) * 0.02 for _ in range(copies)], [r(E, H, ff) * 0.02 for _ in range(copies)]
    turn = [0]

    def at(ws):
        turn[0] += 1
        return ws[turn[0] % len(ws)]

    add(f"router (gemm, fp32 out), {tag}", time_us(lambda: ops.gemm(x, wr, out_dtype=torch.float32)),
        2 * (T * H + wr.numel()) + 4 * logits.numel(), 2.0 * T * wr.numel())
    corr = torch.rand(E, device="cuda") if m.correction else None
    route = lambda: ops.moe_route(logits, E, top, counters, score=m.score, renormalize=m.renormalize, correction=corr)  # noqa: E731
    add(f"moe_route, {tag}", time_us(route), 4 * T * (E + 3 * top))
    rt = route()
    top_i = rt.idx.long()
    add("  vs moe_layout of the homogeneous models", time_us(lambda: moe_ops.moe_layout(top_i, E)), 4 * T * (E + 3 * top))
    pairs, P = T * top, rt.rows
    used = int((torch.bincount(rt.idx.flatten(), minlength=E) > 0).sum())
    xs, scale, h = r(P, H), torch.rand(P, device="cuda"), r(P, ff)
    f = _lib.fn
    add(f"moe_gather, {tag}", time_us(lambda: f("vb_moe_gather")(
        x.data_ptr(), H, rt.dest.data_ptr(), rt.weight.data_ptr(), T, top, H, xs.data_ptr(), scale.data_ptr(), 0, _lib.stream())),
        2 * H * (T + pairs))
    tok, dest = torch.arange(pairs, device="cuda") // top, rt.dest.flatten().long()
    add("  vs index_copy of the homogeneous models", time_us(
        lambda: torch.zeros((P, H), dtype=x.dtype, device="cuda").index_copy(0, dest, x.index_select(0, tok))), 2 * H * (T + pairs))
    add(f"grouped {'gate|up' if m.gated else 'up'}, {tag}", time_us(
        lambda: moe_ops.grouped_product(xs, at(gus), rt.blk_expert), iters=16),
        2 * (pairs * (H + first) + used * first * H), 2.0 * pairs * H * first)
    dense = [r(first * (top if T > 2048 else E), H) * 0.02 for _ in range(copies)]
    add("  vs gemm of that size", time_us(lambda: ops.gemm(x, at(dense)), iters=16),
        2 * (T * (H + dense[0].shape[0]) + dense[0].numel()), 2.0 * T * dense[0].numel())
    del dense
    gu = moe_ops.grouped_product(xs, gus[0], rt.blk_expert)
    if m.gated:
        add(f"silu_glu of the routed rows, {tag}", time_us(lambda: f("vb_silu_glu")(
            gu.data_ptr(), 2 * ff, h.data_ptr(), P, ff, scale.data_ptr(), rt.blk_expert.data_ptr(), 0, _lib.stream())),
            pairs * ff * 6)
    else:
        add(f"activation of the routed rows ({m.act}), {tag}", time_us(
            lambda: ops.activation(gu, ff, m.act, rt.blk_expert)), pairs * ff * 4)
    add(f"grouped down, {tag}", time_us(lambda: moe_ops.grouped_product(h, at(downs), rt.blk_expert), iters=16),
        2 * (pairs * (H + ff) + used * ff * H), 2.0 * pairs * H * ff)
    out = moe_ops.grouped_product(h, downs[0], rt.blk_expert)
    parts = ops.RoutedSum(out, rt, m.weigh == "output", r(T, H), logits[:, E] if m.shared_gate else None)
    if m.shared_gate:
        add(f"moe_combine (+ shared, residual, copy), {tag}", time_us(lambda: ops.moe_combine(parts, res, None, 1e-5)),
            2 * H * (pairs + T) + 10 * T * H)
    else:
        g = r(T, H)
        add(f"moe_norm_add (+ shared, gate, norm, residual, next norm), {tag}", time_us(
            lambda: ops.moe_norm_add(parts, res, w, 1e-5, final_weight=w, gate=g)), 2 * H * (pairs + 2 * T) + 10 * T * H)
    tw = rt.weight.to(x.dtype).unsqueeze(-1)
    add("  vs sum and residual of the homogeneous models", time_us(lambda: ops.rmsnorm(
        (out.index_select(0, dest).view(T, top, H) * tw).sum(1), w, 1e-5, x)), 2 * H * (pairs + T) + 6 * T * H)


def _bench_lru(add, r, m, B: int, n: int, DB: int, ctx: int) -> None:
    T, W = B * n, m.width
    proj, gates = r(T, m.proj_size), r(2 * m.blocks, m.block_size, m.block_size) * m.block_size ** -0.5
    gb, lam = torch.randn(2 * m.blocks, m.block_size, device="cuda"), torch.rand(W, device="cuda") * 6 - 5
    conv, cb, nslot = r(W, m.conv) * 0.5, r(W), max(B, DB)
    ring, state = r(nslot, m.conv, W), torch.zeros(nslot, W, device="cuda")
    sl = torch.arange(nslot, device="cuda", dtype=torch.int32)
    cu = torch.arange(B + 1, device="cuda", dtype=torch.int32) * n
    lens = torch.full((B,), n, device="cuda", dtype=torch.int32)
    add("rglru prefill (conv, gates, recurrence)", time_us(
        lambda: ops.rglru(proj, conv, cb, gates, gb, lam, ring, state, cu, lens, sl[:B], n)),
        T * 3 * W * 2, 4.0 * T * W * m.block_size)
    cu1, lens1 = torch.arange(DB + 1, device="cuda", dtype=torch.int32), torch.full((DB,), ctx, device="cuda", dtype=torch.int32)
    # weights, rings and states rotate, so that they come from memory
    gs, rings, states = [gates.clone() for _ in range(16)], [ring.clone() for _ in range(16)], [state.clone() for _ in range(16)]
    turn = [0]

    def step():
        turn[0] += 1
        i = turn[0] % 16
        return ops.rglru(proj[:DB], conv, cb, gs[i], gb, lam, rings[i], states[i], cu1, lens1, sl[:DB], 1)

    add("rglru decode (conv, fused step)", time_us(step, iters=32),
        2 * gates.numel() + DB * W * (3 * 2 + (m.conv + 1) * 2 + 8), 4.0 * DB * W * m.block_size)


def _bench_delta(add, r, dl, B: int, n: int, DB: int, ctx: int) -> None:
    T = B * n
    cu = torch.arange(B + 1, device="cuda", dtype=torch.int32) * n
    cu1 = torch.arange(DB + 1, device="cuda", dtype=torch.int32)
    proj = r(T, dl.proj_size)
    conv, alog = r(dl.channels, dl.conv) * 0.5, torch.zeros(dl.heads, device="cuda")
    nw, dt = r(dl.vdim), torch.full((dl.heads,), -3.0, device="cuda")
    nslot = max(B, DB)
    ring = r(nslot, dl.conv, dl.channels)
    state = torch.zeros(nslot, dl.heads, dl.vdim, dl.dim, device="cuda")
    sl = torch.arange(nslot, device="cuda", dtype=torch.int32)
    lens = torch.full((B,), n, device="cuda", dtype=torch.int32)
    dims = (dl.heads, dl.kv_heads, dl.dim, dl.vdim, 1e-5)
    add("delta_rule prefill (conv, recurrence, gated norm)", time_us(
        lambda: ops.delta_rule(proj, conv, alog, dt, nw, ring, state, cu, lens, sl[:B], n, *dims)),
        T * (dl.proj_size + dl.out_size) * 2, 6.0 * T * dl.heads * dl.dim * dl.vdim)
    lens = torch.full((DB,), ctx, device="cuda", dtype=torch.int32)
    add("delta_rule decode (fused step)", time_us(
        lambda: ops.delta_rule(proj[:DB], conv, alog, dt, nw, ring, state, cu1, lens, sl[:DB], 1, *dims)),
        DB * (2 * 4 * dl.heads * dl.dim * dl.vdim + (dl.proj_size + dl.out_size + dl.conv * dl.channels) * 2))


def _bench_gla(add, r, m, B: int, n: int, DB: int, ctx: int) -> None:
    T, nslot = B * n, max(B, DB)
    proj = r(T, m.proj_size)
    w, b, nw = r(m.qk_size, m.rank) * m.rank ** -0.5, torch.rand(m.qk_size, device="cuda") * 4, r(m.vdim)
    state = torch.zeros(nslot, m.heads, m.vdim, m.dim, device="cuda")
    sl = torch.arange(nslot, device="cuda", dtype=torch.int32)
    dims = (m.heads, m.dim, m.vdim, m.tau, 1e-5)
    cu = torch.arange(B + 1, device="cuda", dtype=torch.int32) * n
    lens = torch.full((B,), n, device="cuda", dtype=torch.int32)
    add("gated linear attention prefill (chunks, gated norm)", time_us(
        lambda: ops.gated_linear_attention(proj, w, b, nw, state, cu, lens, sl[:B], n, *dims)),
        T * (m.proj_size + m.out_size) * 2, 4.0 * T * m.heads * m.dim * m.vdim)
    cu1, lens1 = torch.arange(DB + 1, device="cuda", dtype=torch.int32), torch.full((DB,), ctx, device="cuda", dtype=torch.int32)
    add("gated linear attention decode (fused step)", time_us(
        lambda: ops.gated_linear_attention(proj[:DB], w, b, nw, state, cu1, lens1, sl[:DB], 1, *dims)),
        DB * (2 * 4 * m.heads * m.dim * m.vdim + (m.proj_size + m.out_size) * 2))


def main(args) -> dict:
    torch.cuda.set_device(0)
    _lib.load(build_if_missing=False)
    L = args.serving_layers
    bw, tf, kind = _peaks()
    out = {"bench": "serving", "dtype": "bf16", "data": "random tokens, random-init weights",
           "peaks": {"hbm_gbs": bw, "bf16_tflops": tf, "kind": kind}, "timer": "CUDA events; inputs larger than L2"}
    prefills, decodes = [(8, 1024), (8, 2048), (2, 8192)], [(16, 2048), (128, 1024), (128, 4096)]
    out["models"] = [bench_model(m, L, prefills, decodes, args.steps if args.steps > 2 else 5)
                     for m in (args.serving, args.serving_vs)]
    if args.serving_kernels:
        out["kernels"] = {f"prefill {b}x{n}, decode {db}x{c}": bench_kernels(args.serving, args.serving_vs, b, n, db, c)
                          for b, n, db, c in ((8, 2048, 128, 2048), (2, 8192, 32, 8192))}
    code, blk, detail = _lib.read_status()
    if code:
        raise RuntimeError(f"a kernel gave up waiting: code {code} (block {blk}, detail {detail})")
    print(json.dumps(out))
    return out
