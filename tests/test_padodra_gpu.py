"""The Padodra design on the GPU: every mechanism's kernels alone, then whole models through the engine, against the plain
implementation in ``_padodra_oracle.py`` (fp32 on the CPU)."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import _padodra_models as M
import _padodra_oracle as O
from verl_b200 import ops
from verl_b200.ops import _lib
from verl_b200.rollout import SamplingParams

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
DTYPES = pytest.mark.parametrize("dtype", [F32, BF], ids=["fp32", "bf16"])


def rand(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def i32(*t):
    return torch.tensor(t, dtype=torch.int32).cuda()


def close(got, want, dtype, f32=2e-5, bf16=1e-2):
    got, want = got.float().cpu(), want.float()
    err = float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp(min=1e-12))
    assert err < (f32 if dtype == F32 else bf16), err
    assert _lib.read_status()[0] == 0


# ------------------------------------------------------------------------------------------------ token-wise mechanisms
@DTYPES
@pytest.mark.parametrize("H", [8, 52, 96, 1000, 4096])
def test_norm_of_the_output_and_embedding(dtype, H):
    x, res, w, fw = rand(37, H, seed=1, dtype=dtype), rand(37, H, seed=2, scale=3.0), rand(H, seed=3, dtype=dtype), rand(
        H, seed=4, dtype=dtype)
    r = res.cuda()
    want = res + O.rms_norm(x.float(), 1e-3, w.float())
    close(ops.rmsnorm_add(x.cuda(), r, w.cuda(), 1e-3), want, dtype)
    close(r, want, F32)
    want2 = want + O.rms_norm(x.float(), 1e-3, w.float())
    y = ops.rmsnorm_add(x.cuda(), r, w.cuda(), 1e-3, final_weight=fw.cuda(), final_scale=0.3)
    close(y, O.rms_norm(want2, 1e-3, fw.float()) * 0.3, dtype)
    close(r, want2, F32)
    table, ids = rand(50, H, seed=4, dtype=dtype), torch.tensor([0, 49, 7, 7])
    res, copy = ops.embedding_scaled(ids.cuda(), table.cuda(), 1.7, with_copy=True)
    close(res, table.float()[ids] * 1.7, F32)
    close(copy, table.float()[ids] * 1.7, dtype)


@DTYPES
@pytest.mark.parametrize("ff", [64, 52, 1024])
def test_gelu_glu(dtype, ff):
    gu = rand(33, 2 * ff + 8, seed=5, dtype=dtype, scale=2.0)
    gu[0, :4] = torch.tensor([-60.0, 60.0, 0.0, -4.0])
    close(ops.gelu_tanh_glu(gu.cuda(), ff), O.gelu_tanh(gu[:, :ff].float()) * gu[:, ff:2 * ff].float(), dtype)


def paged(k, v, bs, seed=0):
    """[n, G, D] -> paged caches with shuffled pages (stale values in the unused places) and the block table row."""
    n, G, D = k.shape
    nb = (n + bs - 1) // bs
    kc, vc = rand(nb + 2, G, bs, D, seed=91, dtype=k.dtype), rand(nb + 2, G, bs, v.shape[2], seed=92, dtype=v.dtype)
    table = torch.randperm(nb + 2, generator=torch.Generator().manual_seed(seed))[:nb].int()
    at = torch.arange(n)
    kc[table[at // bs].long(), :, at % bs], vc[table[at // bs].long(), :, at % bs] = k, v
    return kc.cuda(), vc.cuda(), table.view(1, -1).cuda()


@DTYPES
@pytest.mark.parametrize("H,G,D,V,dims,interleaved", [(4, 2, 32, 24, 32, True), (3, 3, 20, 12, 6, True), (8, 1, 128, 128, 80, True),
                                                      (5, 5, 48, 16, 16, True), (2, 1, 160, 64, 160, True), (4, 2, 32, 32, 24, False),
                                                      (2, 2, 96, 96, 0, True)])
def test_head_norm_rotation_and_cache_write(dtype, H, G, D, V, dims, interleaved):
    T, BS, pos0 = 21, 16, 1000
    n = (H + G) * D + G * V
    qkv, qw, kw = rand(T, n + 8 - n % 8, seed=1, dtype=dtype), rand(D, seed=2, dtype=dtype), rand(D, seed=3, dtype=dtype)
    kc, vc = torch.zeros(5, G, BS, D, dtype=dtype).cuda(), torch.zeros(5, G, BS, V, dtype=dtype).cuda()
    slots = torch.randperm(5 * BS, generator=torch.Generator().manual_seed(1))[:T]
    slots[3] = -1
    freqs = O.llama3_frequencies(dims, 3000.0, M.LLAMA3) if dims else []
    q = ops.head_norm_rope_kv_write(qkv.clone().cuda(), qw.cuda(), kw.cuda(), torch.tensor(freqs).cuda() if dims else None,
                                    torch.arange(pos0, pos0 + T).cuda(), slots.cuda(), kc, vc, H, 1e-2,
                                    interleaved=interleaved, amplitude=1.25)
    f = torch.cat([torch.zeros(pos0, n), qkv[:, :n].float()])

    def turned(x, w):
        x = O.rms_norm(x, 1e-2, w.float())
        return (O.rotate(x, freqs, interleaved, 1.25) if dims else x)[pos0:]

    close(q, turned(f[:, :H * D].view(-1, H, D), qw), dtype, f32=1e-4)
    ok = slots >= 0
    blk, off = slots[ok] // BS, slots[ok] % BS
    close(kc.cpu()[blk, :, off], turned(f[:, H * D:(H + G) * D].view(-1, G, D), kw)[ok], dtype, f32=1e-4)
    close(vc.cpu()[blk, :, off], f[pos0:, (H + G) * D:].view(T, G, V)[ok], dtype, f32=1e-7, bf16=1e-7)
    assert int((kc.abs().amax((1, 3)) > 0).sum()) == T - 1


@DTYPES
@pytest.mark.parametrize("H,N,rot,rank", [(4, 24, 16, 48), (5, 12, 6, 28), (3, 128, 64, 512), (2, 40, 32, 72)])
def test_latent_rotation_norm_and_cache_write(dtype, H, N, rot, rank):
    T, BS, pos0 = 19, 16, 700
    nq = H * (N + rot)
    proj, w = rand(T, (nq + rank + rot + 15) // 8 * 8, seed=1, dtype=dtype), rand(rank, seed=2, dtype=dtype)
    pages = torch.zeros(4, BS, ops.latent_width(rank + rot), dtype=dtype).cuda()
    slots = torch.randperm(4 * BS, generator=torch.Generator().manual_seed(1))[:T]
    slots[5] = -1
    freqs, amp = O.yarn_frequencies(rot, 2000.0, M.YARN)
    assert amp != 1.0
    x = proj.clone().cuda()
    ops.latent_rope_write(x, w.cuda(), torch.tensor(freqs).cuda(), torch.arange(pos0, pos0 + T).cuda(), slots.cuda(), pages, H, N,
                          rot, rank, 1e-2, amplitude=amp)
    f = torch.cat([torch.zeros(pos0, proj.shape[1]), proj.float()])
    q = f[:, :nq].view(-1, H, N + rot)
    want = torch.cat([q[..., :N], O.rotate(q[..., N:], freqs, False, amp)], -1)[pos0:]
    close(x[:, :nq].reshape(T, H, -1), want, dtype, f32=1e-4)
    assert torch.equal(x[:, nq:].cpu(), proj[:, nq:])  # what lies behind the queries stays
    row = torch.cat([O.rms_norm(f[:, nq:nq + rank], 1e-2, w.float()),
                     O.rotate(f[:, nq + rank:nq + rank + rot], freqs, False, amp)], -1)[pos0:]
    flat = pages.view(-1, pages.shape[2]).cpu()
    close(flat[slots[slots >= 0], :rank + rot], row[slots >= 0], dtype, f32=1e-4)
    assert float(flat[:, rank + rot:].abs().sum()) == 0 and int((flat.abs().amax(1) > 0).sum()) == T - 1


# ------------------------------------------------------------------------------------------------------------ attention
@DTYPES
@pytest.mark.parametrize("impl", ["tc", "simt"])
@pytest.mark.parametrize("H,G,D,V,chunk,cap,bs", [
    (4, 2, 48, 40, 50, 3.0, 16), (2, 2, 128, 128, 128, 30.0, 32), (3, 1, 64, 64, 1, 5.0, 16), (2, 1, 16, 128, 130, 0.0, 64),
    (8, 1, 128, 64, 300, 0.7, 16), (2, 2, 8, 8, 1000, 8.0, 8), (2, 1, 32, 32, 0, 4.0, 16)])
def test_attention(dtype, impl, H, G, D, V, chunk, cap, bs):
    if impl == "tc" and dtype == F32:
        pytest.skip("the tensor-core kernels are bf16")
    n = 333
    q, k, v = (rand(n, h, d, seed=s, dtype=dtype) for h, d, s in ((H, D, 1), (G, D, 2), (G, V, 3)))
    gate, sink = rand(n, H * V, seed=4, dtype=dtype, scale=2.0), rand(H, seed=5, scale=3.0)
    mask = O.chunk_mask(n, chunk) if chunk else O.causal_mask(n)
    want = O.attend(q.float(), k.float(), v.float(), 0.4, mask, cap or None, sink).reshape(n, -1)
    kc, vc, bt = paged(k, v, bs)
    for lo, hi in ((0, n), (0, 1), (127, 129), (200, 333), (332, 333), (299, 301)):  # portions, and single tokens
        args = (q[lo:hi].cuda(), kc, vc, bt, i32(0, hi - lo), i32(hi), hi - lo)
        kw = dict(scale=0.4, chunk=chunk, softcap=cap, sink=sink.cuda(), impl=impl)
        close(ops.paged_attention(*args, **kw), want[lo:hi], dtype)
        close(ops.paged_attention(*args, **kw, gate=gate[lo:hi].cuda()), want[lo:hi] * O.sigmoid(gate[lo:hi].float()), dtype)


@DTYPES
@pytest.mark.parametrize("decode", [False, True])
def test_attention_chunk_edges(dtype, decode):
    """One key that outweighs all others is put just inside and just outside of the query's chunk, at page and block borders:
    the output is its value, or has nothing of it."""
    D, bs = 32, 16
    for chunk, rows in ((150, (149, 150, 151, 299, 300)), (128, (127, 128, 129, 256)), (37, (36, 37, 110, 111, 112))):
        for i in rows:
            n, start = i + 1, i // chunk * chunk
            for j in {0, 15, 16, start - 2, start - 1, start, start + 1, i - 1, i, 127, 128, i // 16 * 16, i // 16 * 16 - 1}:
                if not 0 <= j <= i:
                    continue
                q, k, v = torch.zeros(n, 1, D), torch.zeros(n, 1, D), torch.zeros(n, 1, D)
                q[:, 0, 3], k[j, 0, 3], v[j, 0] = 5.0, 6.0, 1.0
                kc, vc, bt = paged(k.to(dtype), v.to(dtype), bs)
                lo = i if decode else max(0, i - 2)
                out = ops.paged_attention(q[lo:].to(dtype).cuda(), kc, vc, bt, i32(0, n - lo), i32(n), n - lo, scale=1.0,
                                          chunk=chunk, softcap=25.0)
                assert abs(float(out[-1].float().mean()) - (1.0 if j >= start else 0.0)) < 1e-2, (chunk, i, j)


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("cap", [0.0, 50.0, 2.0])
def test_attention_large_scores_and_sinks(decode, cap):
    """Scores far apart (the running reference has to move), scores at the cap's ends, sinks above and below all scores."""
    n, D = 300, 64
    q, k, v = rand(n, 4, D, seed=1, dtype=BF, scale=4.0), rand(n, 2, D, seed=2, dtype=BF, scale=4.0), rand(n, 2, D, seed=3, dtype=BF)
    k[::50] *= 3
    kc, vc, bt = paged(k, v, 16)
    lo = n - 1 if decode else 0
    sink = torch.tensor([-200.0, 0.0, 30.0, 90.0])
    for scale in (0.3, -0.3):
        want = O.attend(q.float(), k.float(), v.float(), scale, O.chunk_mask(n, 210), cap or None, sink).reshape(n, 4, D)
        got = ops.paged_attention(q[lo:].cuda(), kc, vc, bt, i32(0, n - lo), i32(n), n - lo, scale=scale, chunk=210, softcap=cap,
                                  sink=sink.cuda()).view(-1, 4, D)
        for h in range(4):  # a head whose sink takes all has next to nothing left: compare in units of the values
            assert float((got[:, h].float().cpu() - want[lo:, h]).pow(2).mean().sqrt()) < 1e-2, (scale, h)
    assert _lib.read_status()[0] == 0


def test_attention_small_scores_keep_their_differences():
    """The cap must not swallow small differences: many keys with scores close to one another under a large cap."""
    n, D = 260, 32
    q, k, v = rand(n, 2, D, seed=1, dtype=BF, scale=0.2), rand(n, 2, D, seed=2, dtype=BF, scale=0.2), rand(n, 2, D, seed=3, dtype=BF)
    kc, vc, bt = paged(k, v, 16)
    for cap in (500.0, 50.0, 4.0, 1.5):  # from far inside the cap to scores on both sides of it
        want = O.attend(q.float(), k.float(), v.float(), 3.0, O.causal_mask(n), cap).reshape(n, -1)
        for lo in (0, n - 1):
            close(ops.paged_attention(q[lo:].cuda(), kc, vc, bt, i32(0, n - lo), i32(n), n - lo, scale=3.0, softcap=cap),
                  want[lo:], BF, bf16=4e-3)


# ----------------------------------------------------------------------------------------------------- latent attention
LATENT_SIZES = pytest.mark.parametrize("H,N,rot,V,rank,bs", [
    (4, 24, 16, 40, 48, 16), (36, 16, 16, 16, 200, 16), (2, 128, 64, 128, 512, 32), (16, 64, 64, 64, 128, 64), (5, 12, 6, 20, 28, 16),
    (33, 32, 8, 32, 136, 8)])


def latent_case(H, N, rot, V, rank, dtype, n=333, gain=1.0):
    width = ops.latent_width(rank + rot)
    rows = torch.zeros(n, width, dtype=dtype)
    rows[:, :rank + rot] = rand(n, rank + rot, seed=1, dtype=dtype)
    q = rand(n, H, N + rot, seed=2, dtype=dtype, scale=gain)
    uk, uv = rand(H, N, rank, seed=3, dtype=dtype, scale=rank ** -0.5), rand(H, V, rank, seed=4, dtype=dtype, scale=rank ** -0.5)
    gate = rand(n, H * V, seed=5, dtype=dtype, scale=2.0)
    return width, rows, q, uk, uv, gate


def latent_oracle(rows, q, uk, uv, scale, rank, rot, gate):
    f = rows.float()
    k = torch.cat([torch.einsum("tr,hnr->thn", f[:, :rank], uk.float()),
                   f[:, None, rank:rank + rot].expand(-1, q.shape[1], -1)], -1)
    v = torch.einsum("tr,hvr->thv", f[:, :rank], uv.float())
    o = O.attend(q.float(), k, v, scale, O.causal_mask(len(f))).reshape(len(f), -1)
    return o * O.sigmoid(gate.float())


def latent_pages(rows, bs):
    kc, _, bt = paged(rows[:, None], rows[:, None], bs)
    return kc[:, 0].contiguous(), bt


@DTYPES
@pytest.mark.parametrize("impl", ["tc", "simt"])
@LATENT_SIZES
def test_latent_attention_in_the_latent_space(dtype, impl, H, N, rot, V, rank, bs):
    if impl == "tc" and (dtype == F32 or N % 8):
        pytest.skip("the tensor-core kernels are bf16, with sizes in multiples of 8")
    n, scale = 333, 0.25
    width, rows, q, uk, uv, gate = latent_case(H, N, rot, V, rank, dtype)
    want = latent_oracle(rows, q, uk, uv, scale, rank, rot, gate)
    pages, bt = latent_pages(rows, bs)
    for lo, hi in ((0, 1), (127, 129), (250, 282), (332, 333), (255, 257)):
        T = hi - lo
        qa = ops.latent_queries(q[lo:hi].cuda(), uk.cuda(), impl=impl)
        close(qa[..., :rank], torch.einsum("thn,hnr->thr", q[lo:hi, :, :N].float(), uk.float()), dtype)
        assert torch.equal(qa[..., rank:rank + rot].cpu(), q[lo:hi, :, N:]) and float(qa[..., rank + rot:].abs().sum()) == 0
        lat = ops.latent_attention(qa, pages, bt, i32(0, T), i32(hi), rank, scale=scale, max_ctx=hi, impl=impl)
        out = torch.empty(T, H * V, dtype=dtype, device="cuda")
        ops.latent_values(lat, uv.cuda(), gate[lo:hi].cuda(), out, impl=impl)
        close(out, want[lo:hi], dtype, bf16=2e-2)


@LATENT_SIZES
def test_latent_attention_expanded(H, N, rot, V, rank, bs):
    if not ops.latent_prefill_supported(H, N, rot, V, rank, BF, "cuda"):
        assert N % 8 or rot % 8
        return
    n, scale = 333, 0.25
    width, rows, q, uk, uv, gate = latent_case(H, N, rot, V, rank, BF)
    want = latent_oracle(rows, q, uk, uv, scale, rank, rot, gate)
    pages, bt = latent_pages(rows, bs)
    up = torch.cat([uk.reshape(-1, rank), uv.reshape(-1, rank)]).cuda()
    # two sequences over the same pages: the whole prompt, and a portion of a shorter one between other tokens' rows
    lo, hi = 150, 290
    ctx = i32(0, n, n + hi)
    both = torch.cat([bt, bt])
    got_rows = ops.latent_gather(pages, both, ctx, n + hi)
    assert torch.equal(got_rows.cpu(), torch.cat([rows, rows[:hi]]))
    kv = ops.gemm(got_rows[:, :rank], up)
    qq, gg = torch.cat([q, q[lo:hi]]).cuda(), torch.cat([gate, gate[lo:hi]]).cuda()
    out = torch.full((n + hi - lo + 3, H * V), 7.0, dtype=BF, device="cuda")
    ops.latent_prefill(qq, got_rows[:, rank:rank + rot], kv, i32(0, n, n + hi - lo), ctx, n, N, V, scale=scale, gate=gg, out=out)
    close(out[:n], want, BF, bf16=2e-2)
    close(out[n:-3], want[lo:hi], BF, bf16=2e-2)
    assert bool((out[-3:] == 7.0).all())


@pytest.mark.parametrize("form", ["latent", "expanded"])
def test_latent_attention_far_keys(form):
    """One key that outweighs all others, anywhere in the context: block, page and split borders, the first and last tokens."""
    H, N, rot, V, rank, n = 2, 16, 16, 16, 64, 700
    for j in (0, 1, 15, 16, 127, 128, 255, 256, 383, 511, 512, 640, 698, 699):
        rows = torch.zeros(n, ops.latent_width(rank + rot), dtype=BF)
        rows[j, rank + 3], rows[j, 5] = 6.0, 1.0       # the rotated part stands out, the latent carries the value
        q = torch.zeros(n, H, N + rot, dtype=BF)
        q[:, :, N + 3] = 5.0
        uk, uv = torch.zeros(H, N, rank, dtype=BF).cuda(), torch.zeros(H, V, rank, dtype=BF).cuda()
        uv[:, :, 5] = 1.0
        pages, bt = latent_pages(rows, 16)
        if form == "latent":
            qa = ops.latent_queries(q[-1:].cuda(), uk)
            lat = ops.latent_attention(qa, pages, bt, i32(0, 1), i32(n), rank, scale=1.0, max_ctx=n)
            out = ops.latent_values(lat, uv, None, torch.empty(1, H * V, dtype=BF, device="cuda"))
        else:
            ctx = i32(0, n)
            r = ops.latent_gather(pages, bt, ctx, n)
            kv = ops.gemm(r[:, :rank], torch.cat([uk.view(-1, rank), uv.view(-1, rank)]))
            out = torch.empty(n, H * V, dtype=BF, device="cuda")
            ops.latent_prefill(q.cuda(), r[:, rank:rank + rot], kv, i32(0, n), ctx, n, N, V, scale=1.0, gate=None, out=out)
            if j > 0:  # the query before it does not see it
                assert abs(float(out[j - 1].float().mean())) < 1e-2, j
        assert abs(float(out[-1].float().mean()) - 1.0) < 1e-2, j
    assert _lib.read_status()[0] == 0


def test_latent_attention_large_scores_and_splits():
    """Scores far apart (references move after the first block) and several splits of a long context, unequal sequences."""
    H, N, rot, V, rank, n = 6, 32, 16, 32, 160, 1500
    width, rows, q, uk, uv, gate = latent_case(H, N, rot, V, rank, BF, n=n, gain=3.0)
    rows[::190, :rank] *= 4
    q = q[:3]
    pages, bt = latent_pages(rows, 16)
    lens = [n, 1, 777]
    qa = ops.latent_queries(q.cuda(), uk.cuda())
    bts = bt.expand(3, -1).contiguous()
    f, want = rows.float(), []
    for x, L in zip(qa.float().cpu(), lens):
        s = x @ f[:L].T * 0.5
        want.append(torch.softmax(s, -1) @ f[:L, :rank])
    for max_ctx in (n, 100000):  # another split count
        got = ops.latent_attention(qa, pages, bts, i32(0, 1, 2, 3), i32(*lens), rank, scale=0.5, max_ctx=max_ctx)
        close(got, torch.stack(want), BF, bf16=5e-3)


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
    for sizes in ([230], [150] + [1] * 80, [33, 2, 64, 1, 1, 17, 3], [2]):  # the same engine: pages again
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
    """Hundreds of decoded tokens: chunks begin among decoded positions, pages are added one by one."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=6)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"))
    ids = tokens(500, cfg["vocab"], 1)
    assert M.error(M.feed_portions(eng, "a", ids, [3] + [1] * 497), O.forward(cfg, w, ids)) < TOL[dtype]


@DTYPES
@pytest.mark.parametrize("short", [1, 32])
def test_unequal_batches(dtype, short, tmp_path):
    """Portions beside single tokens (both forms of latent attention in one step), requests that pause, pages that change
    hands: each as if alone."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=2)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"), num_blocks=28, max_model_len=320)
    eng.model.latent_short = max(short, eng.model.latent_short) if dtype == F32 else short
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
                                {"num_blocks": 10, "enable_prefix_caching": False}])
def test_greedy_generation(kw, tmp_path):
    """generate() with its scheduler: CUDA graphs and bursts, eager steps, portions of prompts, preemption."""
    cfg = M.config([M.attention(2, 1, 32, 32, 23, ff=64), M.latent(2, 16, 16, 32, 32)], vocab=64, width=64)
    w = M.weights(cfg, seed=5)
    eng = M.engine(M.load_model(cfg, w, tmp_path, F32, "cuda"), max_model_len=96, **kw)
    prompts = [tokens(n, 64, n) for n in (21, 5, 33, 14)]
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))
    assert [o.token_ids for o in outs] == [greedy(cfg, w, p, 40) for p in prompts]
    if "num_blocks" in kw:
        assert sum(o.num_preempted for o in outs) > 0


def test_shared_prompts_use_the_prefix_cache(tmp_path):
    cfg = M.config([M.attention(2, 1, 32, 32, 40, ff=64), M.latent(2, 16, 16, 32, 32)], vocab=64, width=64)
    w = M.weights(cfg, seed=5)
    eng = M.engine(M.load_model(cfg, w, tmp_path, F32, "cuda"))
    p = tokens(90, 64)
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    first = eng.generate([p], sp)[0].token_ids
    assert first == greedy(cfg, w, p, 8)
    assert eng.generate([p, p[:70] + [1, 2, 3]], sp)[0].token_ids == first and eng.sched.stats()["prefix_hits"] > 0


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


def test_fp8_weights(tmp_path):
    """rollout.quantization = fp8: coarse, but the same model."""
    cfg = M.config([M.attention(2, 1, 64, 64, 40, ff=128), M.latent(2, 64, 64, 64, 128, ff=128)], vocab=256, width=128)
    w = M.weights(cfg, seed=5)
    eng = M.engine(M.load_model(cfg, w, tmp_path, BF, "cuda"), quantization="fp8")
    ids = tokens(100, 256)
    assert M.error(M.feed_portions(eng, "a", ids, [60, 1, 39]), O.forward(cfg, w, ids)) < 0.6


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
