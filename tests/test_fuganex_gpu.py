"""The Fuganex design on the GPU: every mechanism's kernels alone, then whole models through the engine, against the plain
implementation in ``_fuganex_oracle.py`` (fp32 on the CPU)."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import _fuganex_models as M
import _fuganex_oracle as O
from verl_b200 import ops
from verl_b200.models.layer_specs import distance_buckets
from verl_b200.ops import _lib
from verl_b200.rollout import SamplingParams

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
DTYPES = pytest.mark.parametrize("dtype", [F32, BF], ids=["fp32", "bf16"])


def rand(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got, want, dtype, f32=2e-5, bf16=1e-2):
    got, want = got.float().cpu(), want.float()
    err = float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp(min=1e-12))
    assert err < (f32 if dtype == F32 else bf16), err
    assert _lib.read_status()[0] == 0


# ------------------------------------------------------------------------------------------------ token-wise mechanisms
@DTYPES
@pytest.mark.parametrize("H", [8, 52, 96, 1000, 4096])
def test_norm_embedding(dtype, H):
    x, res, w = rand(37, H, seed=1, dtype=dtype), rand(37, H, seed=2, scale=3.0), rand(H, seed=3, dtype=dtype)
    r = res.cuda()
    y = ops.add_rmsnorm(x.cuda(), r, w.cuda(), 1e-3)
    close(r, res + x.float(), F32)
    close(y, O.rms_norm(res + x.float(), 1e-3, w.float()), dtype)
    close(ops.add_rmsnorm(None, r, w.cuda(), 1e-3), O.rms_norm(res + x.float(), 1e-3, w.float()), dtype)
    table, ids = rand(50, H, seed=4, dtype=dtype), torch.tensor([0, 49, 7, 7])
    close(ops.embedding_scaled(ids.cuda(), table.cuda(), 1.7), table.float()[ids] * 1.7, F32)


@DTYPES
@pytest.mark.parametrize("ff,limit", [(64, 0.5), (52, 1.0), (1024, 7.0)])
def test_clamped_glu(dtype, ff, limit):
    gu = rand(33, 2 * ff + 8, seed=5, dtype=dtype, scale=2.0)
    gu[0, :4], gu[0, ff:ff + 4] = limit, -limit
    gu[1, :2] = torch.tensor([-60.0, 60.0])  # far ends of the sigmoid
    close(ops.clamped_glu(gu.cuda(), ff, limit, 1.702), O.clamped_glu(gu[:, :ff].float(), gu[:, ff:2 * ff].float(), limit), dtype)


@pytest.mark.parametrize("M_,N,K", [(1, 8, 52), (5, 203, 60), (130, 70, 33), (64, 64, 512)])
def test_simt_gemm(M_, N, K):
    a, b = rand(M_, K, seed=1), rand(N, K, seed=2)
    close(ops.gemm(a.cuda(), b.cuda()), a @ b.T, F32, f32=2e-6)  # true fp32, no reduced-precision mode
    if K % 8:
        a, b = a.to(BF), b.to(BF)
        close(ops.gemm(a.cuda(), b.cuda(), out_dtype=F32), a.float() @ b.float().T, F32, f32=1e-5)


@DTYPES
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 32, 24), (3, 3, 20, 12), (8, 1, 128, 128)])
def test_whole_projection_norm_and_cache_write(dtype, H, G, D, V):
    T, BS = 21, 16
    n = H * D + G * D + G * V
    qkv, qw, kw = rand(T, n + 8 - n % 8, seed=1, dtype=dtype), rand(H * D, seed=2, dtype=dtype), rand(G * D, seed=3, dtype=dtype)
    kc, vc = torch.zeros(5, G, BS, D, dtype=dtype).cuda(), torch.zeros(5, G, BS, V, dtype=dtype).cuda()
    slots = torch.randperm(5 * BS, generator=torch.Generator().manual_seed(1))[:T]
    slots[3] = -1
    q = ops.qk_norm_kv_write(qkv.clone().cuda(), qw.cuda(), kw.cuda(), slots.cuda(), kc, vc, H, 1e-4)
    f = qkv.float()
    close(q.reshape(T, -1), O.rms_norm(f[:, :H * D], 1e-4, qw.float()), dtype)
    ok = slots >= 0
    k = O.rms_norm(f[:, H * D:(H + G) * D], 1e-4, kw.float())[ok].view(-1, G, D)
    v = f[:, (H + G) * D:(H + G) * D + G * V][ok].view(-1, G, V)
    blk, off = slots[ok] // BS, slots[ok] % BS
    close(kc.cpu()[blk, :, off], k, dtype)
    close(vc.cpu()[blk, :, off], v, dtype, f32=1e-7, bf16=1e-7)
    assert int((kc.abs().amax((1, 3)) > 0).sum()) == T - 1


# ------------------------------------------------------------------------------------------------------------ attention
def paged(k, v, bs, seed=0):
    """[n, G, D] -> paged caches with shuffled pages (stale values in the unused places) and the block table row."""
    n, G, D = k.shape
    nb = (n + bs - 1) // bs
    kc, vc = rand(nb + 2, G, bs, D, seed=91, dtype=k.dtype), rand(nb + 2, G, bs, v.shape[2], seed=92, dtype=v.dtype)
    table = torch.randperm(nb + 2, generator=torch.Generator().manual_seed(seed))[:nb].int()
    for j in range(n):
        kc[table[j // bs], :, j % bs], vc[table[j // bs], :, j % bs] = k[j], v[j]
    return kc.cuda(), vc.cuda(), table.view(1, -1).cuda()


def oracle_attention(q, k, v, scale, rel, far, window, keep):
    s = O.attention_scores(q.float(), k.float(), scale, rel, far, window, keep)
    rep = q.shape[1] // k.shape[1]
    return torch.einsum("hqk,khd->qhd", torch.softmax(s, -1), v.float().repeat_interleave(rep, 1))


@DTYPES
@pytest.mark.parametrize("impl", ["tc", "simt"])
@pytest.mark.parametrize("H,G,D,V,window,keep,bs", [
    (4, 2, 48, 40, 50, 7, 16), (2, 2, 128, 128, 128, 0, 32), (3, 1, 64, 64, 1, 0, 16), (2, 1, 16, 128, 130, 129, 64),
    (8, 1, 128, 64, 300, 5, 16), (2, 2, 8, 8, 1000, 3, 8)])
def test_attention(dtype, impl, H, G, D, V, window, keep, bs):
    if impl == "tc" and dtype == F32:
        pytest.skip("the tensor-core kernels are bf16")
    n, rows, far = 333, 9, 60
    q, k, v = (rand(n, h, d, seed=s, dtype=dtype) for h, d, s in ((H, D, 1), (G, D, 2), (G, V, 3)))
    rel = rand(rows, H, seed=4)
    want = oracle_attention(q, k, v, 0.3, rel, far, window, keep).reshape(n, -1)
    kc, vc, bt = paged(k, v, bs)
    bias = rel.T[:, torch.tensor(distance_buckets(rows, far))].contiguous().cuda()
    kw = dict(scale=0.3, window=window, keep_first=keep, bias=bias, impl=impl)
    for lo, hi in ((0, n), (0, 1), (127, 129), (200, 333), (332, 333)):  # portions of the prompt, and single tokens
        got = ops.paged_attention(q[lo:hi].cuda(), kc, vc, bt, torch.tensor([0, hi - lo], dtype=torch.int32).cuda(),
                                  torch.tensor([hi], dtype=torch.int32).cuda(), hi - lo, **kw)
        close(got, want[lo:hi], dtype)


@DTYPES
@pytest.mark.parametrize("decode", [False, True])
def test_attention_edges(dtype, decode):
    """One key that outweighs all others is put just inside and just outside of the window and of the kept first tokens, at
    page and chunk borders: the output is its value, or has nothing of it."""
    D, window, keep, bs = 32, 150, 17, 16
    for i in (149, 150, 151, 166, 167, 255, 256, 299):
        n = i + 1
        for j in {0, 15, 16, 17, 18, i - 151, i - 150, i - 149, i - 148, i - 1, i, 127, 128, i // 16 * 16, i // 16 * 16 - 1}:
            if not 0 <= j <= i:
                continue
            q, k, v = torch.zeros(n, 1, D), torch.zeros(n, 1, D), torch.zeros(n, 1, D)
            q[:, 0, 3], k[j, 0, 3], v[j, 0] = 5.0, 6.0, 1.0
            q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
            kc, vc, bt = paged(k, v, bs)
            lo = i if decode else max(0, i - 2)
            out = ops.paged_attention(q[lo:].cuda(), kc, vc, bt, torch.tensor([0, n - lo], dtype=torch.int32).cuda(),
                                      torch.tensor([n], dtype=torch.int32).cuda(), n - lo, scale=1.0, window=window,
                                      keep_first=keep)
            got = float(out[-1].float().mean())
            assert abs(got - (1.0 if O.visible(i, j, window, keep) else 0.0)) < 1e-2, (i, j, got)


def test_attention_bias_reaches_every_distance():
    """Equal scores: the weights are the softmax of the biases alone; every bucket edge shows."""
    n, rows, far, D = 200, 10, 77, 16
    rel = rand(rows, 2, seed=8, scale=2.0)
    bias = rel.T[:, torch.tensor(distance_buckets(rows, far))].contiguous().cuda()
    k, v = torch.zeros(n, 2, D, dtype=BF), rand(n, 2, D, seed=9, dtype=BF)
    q = rand(n, 2, D, dtype=BF)
    kc, vc, bt = paged(k, v, 16)
    for lo in (0, n - 1):
        got = ops.paged_attention(q[lo:].cuda(), kc, vc, bt, torch.tensor([0, n - lo], dtype=torch.int32).cuda(),
                                  torch.tensor([n], dtype=torch.int32).cuda(), n - lo, scale=7.0, window=0, bias=bias)
        close(got, oracle_attention(q, k, v, 7.0, rel, far, 10 ** 6, 0).reshape(n, -1)[lo:], BF)


def test_attention_large_scores():
    """Scores far apart (the running reference has to move) and a negative scale."""
    n, D = 300, 64
    q, k, v = rand(n, 2, D, seed=1, dtype=BF, scale=4.0), rand(n, 2, D, seed=2, dtype=BF, scale=4.0), rand(n, 2, D, seed=3, dtype=BF)
    k[::50] *= 3
    kc, vc, bt = paged(k, v, 16)
    cu, lens = torch.tensor([0, n], dtype=torch.int32).cuda(), torch.tensor([n], dtype=torch.int32).cuda()
    rel = torch.zeros(4, 2)
    for scale in (0.3, -0.3):
        got = ops.paged_attention(q.cuda(), kc, vc, bt, cu, lens, n, scale=scale, window=200, keep_first=2)
        close(got, oracle_attention(q, k, v, scale, rel, 50, 200, 2).reshape(n, -1), BF)


# ----------------------------------------------------------------------------------------------------------- delta rule
def oracle_delta(proj, cw, a_log, dt_bias, nw, H, G, D, V, eps):
    """The mixer between its two projections for one sequence from its start, fp32."""
    q, k, v, gate, b, a = proj[:, :2 * G * D + 2 * H * V + 2 * H].split([G * D, G * D, H * V, H * V, H, H], 1)
    cq, ck, cv = cw.split([G * D, G * D, H * V])
    T = proj.shape[0]
    q, k = O.unit(O.causal_conv_silu(q, cq).view(T, G, D)) * D ** -0.5, O.unit(O.causal_conv_silu(k, ck).view(T, G, D))
    v = O.causal_conv_silu(v, cv).view(T, H, V)
    beta = torch.sigmoid(b)
    g = torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(a + dt_bias, threshold=80.0))
    o, S = zip(*[O.delta_recurrence(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], beta[:, h], g[:, h]) for h in range(H)])
    o = O.rms_norm(torch.stack(o, 1), eps, nw) * O.silu(gate.reshape(T, H, V))
    return o.reshape(T, -1), torch.stack(S).transpose(1, 2)


@pytest.mark.parametrize("dtype,impl", [(F32, "scan"), (BF, "scan"), (BF, "chunk")])
@pytest.mark.parametrize("H,G,D,V,taps", [(6, 2, 56, 24, 4), (2, 2, 40, 72, 3), (3, 1, 128, 128, 1), (2, 1, 96, 136, 8),
                                          (5, 5, 12, 20, 2), (1, 1, 200, 256, 5)])
def test_delta_rule(dtype, impl, H, G, D, V, taps):
    """A whole prompt, portions down to two tokens and single tokens give the same outputs and state; the state slots hold
    other sequences' leftovers before, and neighbours in the batch do not matter."""
    if impl == "chunk" and (D % 8 or V % 8 or D > 128):
        pytest.skip("sizes of the token-by-token scan")
    T, C = 210, 2 * G * D + H * V
    proj = rand(T, (C + H * V + 2 * H + 7) // 8 * 8, seed=1, dtype=dtype)
    cw, nw = rand(C, taps, seed=2, dtype=dtype, scale=taps ** -0.5), rand(V, seed=3, dtype=dtype)
    a_log, dt = rand(H, seed=4), rand(H, seed=5) - 3
    want, S = oracle_delta(proj.float(), cw.float(), a_log, dt, nw.float(), H, G, D, V, 1e-5)
    fixed = [t.cuda() for t in (cw, a_log, dt, nw)]
    ring, state = rand(3, taps, C, seed=6, dtype=dtype).cuda(), rand(3, H, V, D, seed=7).cuda()
    other = rand(150, proj.shape[1], seed=8, dtype=dtype)
    for sizes in ([210], [64, 2, 63, 65, 16], [1, 1, 2, 140, 33, 1, 1, 31], [1] * 210):
        at, outs, left = 0, [], 0
        for n in sizes:
            x, counts, lens, slots = proj[at:at + n], [n], [at + n], [1]
            m = min(150 - left, n) if n > 1 else 0
            if m:  # a second sequence in front
                x, counts, lens, slots = torch.cat([other[left:left + m], x]), [m, n], [left + m, at + n], [2, 1]
                left += m
            i32 = lambda t: torch.tensor(t, dtype=torch.int32).cuda()  # noqa: E731
            o = ops.delta_rule(x.cuda(), *fixed, ring, state, i32(np.cumsum([0] + counts)), i32(lens), i32(slots), max(counts), H,
                               G, D, V, 1e-5, impl=impl)
            outs.append(o[-n:].cpu())
            at += n
        close(torch.cat(outs), want, dtype)
        close(state[1], S, dtype, bf16=4e-3)


@pytest.mark.parametrize("impl", ["scan", "chunk"])
def test_delta_rule_extremes(impl):
    """Decays from almost 1 to almost 0 and steps near 0 and 1, keys that repeat (the correction term matters)."""
    H, G, D, V, T = 2, 1, 64, 64, 200
    C = 2 * G * D + H * V
    proj = rand(T, C + H * V + 2 * H + 4, seed=1, dtype=BF)
    proj[:, G * D:2 * G * D] = proj[:1, G * D:2 * G * D]           # the same key throughout
    proj[:, C + H * V:C + H * V + H] = torch.tensor([8.0, -8.0])   # beta near 1 and near 0
    proj[60:70, C + H * V + H:] = 40.0                             # decays to (almost) nothing
    cw = torch.zeros(C, 2, dtype=BF)
    cw[:, 1] = 1.0
    a_log, dt, nw = torch.tensor([0.0, 2.0]), torch.tensor([-9.0, -4.0]), torch.ones(V, dtype=BF)
    want, S = oracle_delta(proj.float(), cw.float(), a_log, dt, nw.float(), H, G, D, V, 1e-5)
    ring, state = torch.zeros(1, 2, C, dtype=BF).cuda(), torch.zeros(1, H, V, D).cuda()
    i32 = lambda *t: torch.tensor(t, dtype=torch.int32).cuda()  # noqa: E731
    o = ops.delta_rule(proj.cuda(), cw.cuda(), a_log.cuda(), dt.cuda(), nw.cuda(), ring, state, i32(0, T), i32(T), i32(0), T, H, G,
                       D, V, 1e-5, impl=impl)
    close(o, want, BF)
    close(state[0], S, BF, bf16=4e-3)


# --------------------------------------------------------------------------------------------------------- whole models
TOL = {F32: 2e-4, BF: 0.06}


@DTYPES
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_model_portions(name, dtype, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, seed=3)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"))
    ids = tokens(230, cfg["vocab"], 4)
    want = O.forward(cfg, w, ids)
    for sizes in ([230], [150] + [1] * 80, [33, 2, 64, 1, 1, 17, 3], [2]):  # the same engine: pages and slots again
        assert M.error(M.feed_portions(eng, "a", ids, sizes), want) < TOL[dtype], sizes
    assert eng.sched.stats()["free_pages"] == eng.num_blocks and _lib.read_status()[0] == 0


@DTYPES
def test_layers_one_by_one(dtype, tmp_path):
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=3)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"))
    ids = tokens(70, cfg["vocab"], 4)
    _, streams = O.forward(cfg, w, ids, keep_layers=True)
    seen = []
    eng.observe_layers = lambda i, x: seen.append(x.cpu())
    eng.feed([("a", ids, [])], ["a"])
    assert len(seen) == len(streams)
    for a, b in zip(seen, streams):
        assert float((a - b).pow(2).mean().sqrt() / b.std()) < (1e-5 if dtype == F32 else 0.03)


@DTYPES
def test_long_decoding(dtype, tmp_path):
    """Hundreds of decoded tokens: windows and kept tokens pass over decoded positions, pages are added one by one."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=6)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"))
    ids = tokens(500, cfg["vocab"], 1)
    assert M.error(M.feed_portions(eng, "a", ids, [3] + [1] * 497), O.forward(cfg, w, ids)) < TOL[dtype]


@DTYPES
def test_unequal_batches(dtype, tmp_path):
    """Portions beside single tokens, requests that pause, pages and slots that change hands: each as if alone."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=2)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"), num_blocks=28, max_model_len=320)
    lens = {"a": 210, "b": 40, "c": 5, "d": 97, "e": 130, "f": 64, "g": 17}
    ids = {r: tokens(n, cfg["vocab"], k) for k, (r, n) in enumerate(lens.items())}
    want = {r: O.forward(cfg, w, t) for r, t in ids.items()}
    rng = np.random.default_rng(0)
    at, live, waiting = dict.fromkeys(ids, 0), [], list(ids)
    while live or waiting:
        while waiting and len(live) < 4 and sum((lens[r] + 15) // 16 for r in live + waiting[:1]) <= 28:
            live.append(waiting.pop(0))
        step = [r for r in live if rng.random() < 0.8] or live[:1]
        entries, rows, end = [], [], []
        for r in step:
            n = min(int(rng.choice([1, 1, 1, 2, 3, 31, 64, 70])), lens[r] - at[r])
            entries.append((r, ids[r][at[r]:at[r] + n], list(range(n))))
            rows.append(want[r][at[r]:at[r] + n])
            at[r] += n
            if at[r] == lens[r]:
                end.append(r)
        assert M.error(eng.feed(entries, end), torch.cat(rows)) < TOL[dtype], [(r, at[r]) for r in step]
        live = [r for r in live if r not in end]
    assert eng.sched.stats()["free_pages"] == eng.num_blocks


def test_results_do_not_depend_on_company(tmp_path):
    """bf16: the same request alone and in batches differs by rounding only (far below the error against fp32)."""
    cfg = M.CONFIGS["mixed"]
    eng = M.engine(M.load_model(cfg, M.weights(cfg, seed=2), tmp_path, BF, "cuda"))
    ids, other = tokens(100, cfg["vocab"], 1), tokens(220, cfg["vocab"], 2)
    alone = M.feed_portions(eng, "a", ids, [100])
    got = eng.feed([("x", other[:130], []), ("a", ids, list(range(100))), ("y", other[:2], [])], ["a"]).cpu()
    assert M.error(got, alone) < TOL[BF] / 4
    assert M.error(M.feed_portions(eng, "b", ids, [7]), alone) < TOL[BF]


def greedy(cfg, w, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("kw", [{}, {"enforce_eager": True, "decode_burst": 1}, {"max_num_batched_tokens": 32},
                                {"num_blocks": 10}])
def test_greedy_generation(kw, tmp_path):
    """generate() with its scheduler: CUDA graphs and bursts, eager steps, portions of prompts, preemption."""
    cfg = M.config([M.delta(2, 1, 32, 32, 3), M.attention(2, 1, 32, 32, 9, 2, bias_max=20, ff=64)], vocab=64, width=64)
    w = M.weights(cfg, seed=5)
    eng = M.engine(M.load_model(cfg, w, tmp_path, F32, "cuda"), max_model_len=96, **kw)
    prompts = [tokens(n, 64, n) for n in (21, 5, 33, 14)]
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))
    assert [o.token_ids for o in outs] == [greedy(cfg, w, p, 40) for p in prompts]
    if "num_blocks" in kw:
        assert sum(o.num_preempted for o in outs) > 0


def test_generation_in_bf16_follows_its_own_logits(tmp_path):
    """The tokens that generate() picks are the arg-max of the logits that feed() gives for the same sequence, unless two
    logits are within rounding of each other."""
    cfg = M.CONFIGS["mixed"]
    eng = M.engine(M.load_model(cfg, M.weights(cfg, seed=9), tmp_path, BF, "cuda"))
    prompts = [tokens(n, cfg["vocab"], n) for n in (45, 3, 130)]
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=50, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = M.feed_portions(eng, "r", p + o.token_ids[:-1], [len(p) + 49])[len(p) - 1:]
        picked = lg.gather(1, torch.tensor(o.token_ids)[:, None])[:, 0]
        assert float((lg.max(1).values - picked).max() / lg.std()) < TOL[BF]


def test_sleep_and_wake(tmp_path):
    cfg = M.CONFIGS["delta_only"]
    eng = M.engine(M.load_model(cfg, M.weights(cfg), tmp_path, BF, "cuda"))
    ids = tokens(50, cfg["vocab"])
    a = M.feed_portions(eng, "a", ids, [50])
    eng.sleep()
    assert eng.state_cache is None
    eng.wake_up()
    assert torch.equal(M.feed_portions(eng, "a", ids, [50]), a)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run(dtype, tmp_path):
    cfg = M.CONFIGS["odd"]
    w = M.weights(cfg, seed=1)
    model = M.save(cfg, w, tmp_path / "m")
    ids = tokens(60, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[40:41], "want": []}, {"id": "b", "tokens": ids[:7], "want": [6]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[41:], "want": [18, 0]}], "end": ["a"]}]
    repo = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(repo, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out",
                        str(tmp_path / "out"), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.forward(cfg, w, ids)
    for n, rows in ((0, [0, 39]), (1, [6]), (2, [59, 41])):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", "<f4").reshape(len(rows), -1))
        assert M.error(got, want[rows]) < (2e-4 if dtype == "float32" else 0.06)
