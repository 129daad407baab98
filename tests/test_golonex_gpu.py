"""The Golonex design on the GPU: every mechanism's kernels alone, then whole models through the engine, against the plain
implementation in ``_golonex_oracle.py`` (fp32 on the CPU)."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import _golonex_models as M
import _golonex_oracle as O
from verl_b200 import ops
from verl_b200.ops import _lib
from verl_b200.ops import moe as moe_ops
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
def test_normed_embedding_and_copies_of_the_stream(dtype, H):
    table, w, ids = rand(50, H, seed=4, dtype=dtype, scale=0.2), rand(H, seed=3, dtype=dtype), torch.tensor([0, 49, 7, 7])
    close(ops.embedding_normed(ids.cuda(), table.cuda(), w.cuda(), 1e-2), O.rms_norm(table.float()[ids], 1e-2, w.float()), F32)
    res, d = rand(33, H, seed=1, scale=3.0), rand(33, H, seed=2, dtype=dtype)
    r = res.cuda()
    close(ops.add_rmsnorm(d.cuda(), r, None, 1e-2, dtype), res + d.float(), dtype)
    close(r, res + d.float(), F32)
    close(ops.add_rmsnorm(None, r, None, 1e-2, dtype), res + d.float(), dtype)


@DTYPES
@pytest.mark.parametrize("ff", [64, 52, 1024])
def test_silu_glu_and_gelu_rows(dtype, ff):
    gu = rand(33, 2 * ff + 8, seed=5, dtype=dtype, scale=2.0)
    gu[0, :4] = torch.tensor([-60.0, 60.0, 0.0, -4.0])
    close(ops.silu_glu(gu.cuda(), ff), O.silu(gu[:, :ff].float()) * gu[:, ff:2 * ff].float(), dtype)
    table, ids = rand(20, 3 * ff, seed=6, dtype=dtype), torch.randint(0, 20, (33,), generator=torch.Generator().manual_seed(0))
    for i in range(3):
        got = ops.gelu_rows(gu[:, :ff].cuda(), ids.cuda(), table.cuda(), i * ff, ff)
        close(got, O.gelu_tanh(gu[:, :ff].float()) * table.float()[ids, i * ff:(i + 1) * ff], dtype)


@pytest.mark.parametrize("n", [(3, 331), (5, 64)])
def test_softcap_of_logits(n):
    x = rand(*n, scale=30.0)
    x[0, :3] = torch.tensor([1e4, -1e4, 1e-3])
    close(ops.softcap_(x.clone().cuda(), 7.5), 7.5 * torch.tanh(x / 7.5), F32, f32=1e-6)


@DTYPES
@pytest.mark.parametrize("H,G,D,dims", [(4, 2, 32, 32), (3, 3, 20, 6), (8, 1, 128, 80), (2, 1, 160, 64), (6, 2, 48, 8)])
def test_rotation_and_values_that_are_the_keys(dtype, H, G, D, dims):
    T, BS, pos0 = 21, 16, 1000
    n = (H + G) * D
    qk = rand(T, n + 8 - n % 8, seed=1, dtype=dtype)
    kc, vc = (torch.zeros(5, G, BS, D, dtype=dtype).cuda() for _ in range(2))
    slots = torch.randperm(5 * BS, generator=torch.Generator().manual_seed(1))[:T]
    slots[3] = -1
    freqs, amp = O.yarn_frequencies(dims, 3000.0, M.YARN)
    x = qk.clone().cuda()
    q = ops.head_norm_rope_kv_write(x, None, None, torch.tensor(freqs).cuda(), torch.arange(pos0, pos0 + T).cuda(), slots.cuda(), kc,
                                    vc, H, 1e-6, interleaved=True, amplitude=amp, key_values=True)
    f = torch.cat([torch.zeros(pos0, n), qk[:, :n].float()])
    close(q, O.rotate(f[:, :H * D].view(-1, H, D), freqs, True, amp)[pos0:], dtype, f32=1e-4)
    k = f[:, H * D:].view(-1, G, D)
    ok = slots >= 0
    blk, off = slots[ok] // BS, slots[ok] % BS
    close(kc.cpu()[blk, :, off], O.rotate(k, freqs, True, amp)[pos0:][ok], dtype, f32=1e-4)
    assert torch.equal(vc.cpu()[blk, :, off].float(), k[pos0:][ok])  # as projected
    assert torch.equal(x[:, H * D:].cpu(), qk[:, H * D:]) and int((kc.abs().amax((1, 3)) > 0).sum()) == T - 1


@DTYPES
@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("H,N,rot,rank,q_rank", [(4, 24, 16, 48, 56), (5, 12, 6, 28, 34), (3, 128, 64, 512, 1536), (2, 40, 8, 72, 8)])
def test_latents_of_queries_and_keys(dtype, interleaved, H, N, rot, rank, q_rank):
    T, BS, pos0 = 19, 16, 700
    proj, w, qw = rand(T, (q_rank + rank + rot + 15) // 8 * 8, seed=1, dtype=dtype), rand(rank, seed=2, dtype=dtype), rand(
        q_rank, seed=3, dtype=dtype)
    pages = torch.zeros(4, BS, ops.latent_width(rank + rot), dtype=dtype).cuda()
    slots = torch.randperm(4 * BS, generator=torch.Generator().manual_seed(1))[:T]
    slots[5] = -1
    freqs, amp = O.yarn_frequencies(rot, 2000.0, M.YARN)
    turn = dict(amplitude=amp, interleaved=interleaved)
    x, pos = proj.clone().cuda(), torch.arange(pos0, pos0 + T).cuda()
    ops.latent_rope_write(x, w.cuda(), torch.tensor(freqs).cuda(), pos, slots.cuda(), pages, 0, N, rot, rank, 1e-2, **turn,
                          q_rank=q_rank, q_norm_w=qw.cuda())
    f = proj.float()
    close(x[:, :q_rank], O.rms_norm(f[:, :q_rank], 1e-2, qw.float()), dtype)
    assert torch.equal(x[:, q_rank:].cpu(), proj[:, q_rank:])
    key = torch.cat([torch.zeros(pos0, rot), f[:, q_rank + rank:q_rank + rank + rot]])
    row = torch.cat([O.rms_norm(f[:, q_rank:q_rank + rank], 1e-2, w.float()), O.rotate(key, freqs, interleaved, amp)[pos0:]], -1)
    flat = pages.view(-1, pages.shape[2]).cpu()
    close(flat[slots[slots >= 0], :rank + rot], row[slots >= 0], dtype, f32=1e-4)
    assert float(flat[:, rank + rot:].abs().sum()) == 0 and int((flat.abs().amax(1) > 0).sum()) == T - 1
    # the queries' tails
    nq = H * (N + rot)
    q = rand(T, (nq + 7) // 8 * 8 + 8, seed=7, dtype=dtype)
    y = q.clone().cuda()
    ops.rotate_tails(y, torch.tensor(freqs).cuda(), pos, H, N, rot, **turn)
    full = torch.cat([torch.zeros(pos0, H, N + rot), q[:, :nq].float().view(T, H, -1)])
    want = torch.cat([full[..., :N], O.rotate(full[..., N:], freqs, interleaved, amp)], -1)[pos0:]
    close(y[:, :nq].reshape(T, H, -1), want, dtype, f32=1e-4)
    assert torch.equal(y[:, nq:].cpu(), q[:, nq:])


# ------------------------------------------------------------------------------------------------------------ attention
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
@pytest.mark.parametrize("H,G,D,window", [(6, 3, 32, 37), (8, 1, 64, 128), (16, 1, 16, 141), (4, 4, 128, 1), (2, 1, 48, 500)])
def test_attention_with_a_window(dtype, H, G, D, window):
    n = 333
    q, k, v = (rand(n, h, D, seed=s, dtype=dtype) for h, s in ((H, 1), (G, 2), (G, 3)))
    want = O.attend(q.float(), k.float(), v.float(), 0.4, O.window_mask(n, window)).reshape(n, -1)
    kc, vc, bt = paged(k, v, 16)
    for lo, hi in ((0, n), (0, 1), (127, 129), (200, 333), (332, 333)):
        got = ops.paged_attention(q[lo:hi].cuda(), kc, vc, bt, i32(0, hi - lo), i32(hi), hi - lo, scale=0.4, window=window)
        close(got, want[lo:hi], dtype)


@DTYPES
@pytest.mark.parametrize("decode", [False, True])
def test_attention_window_edges(dtype, decode):
    """One key that outweighs all others just inside and just outside of the window, at page and block borders, at the
    sequence's first tokens: the output is its value, or has nothing of it."""
    D, bs = 32, 16
    for window, rows in ((50, (49, 50, 51, 300)), (128, (127, 128, 129, 255, 256)), (129, (128, 129, 260)), (1, (0, 77))):
        for i in rows:
            n, edge = i + 1, i - window + 1
            for j in {0, 1, 15, 16, edge - 1, edge, edge + 1, i - 1, i, 127, 128, i // 16 * 16, i // 16 * 16 - 1}:
                if not 0 <= j <= i:
                    continue
                q, k, v = torch.zeros(n, 1, D), torch.zeros(n, 1, D), torch.zeros(n, 1, D)
                q[:, 0, 3], k[j, 0, 3], v[j, 0] = 5.0, 6.0, 1.0
                kc, vc, bt = paged(k.to(dtype), v.to(dtype), bs)
                lo = i if decode else max(0, i - 2)
                out = ops.paged_attention(q[lo:].to(dtype).cuda(), kc, vc, bt, i32(0, n - lo), i32(n), n - lo, scale=1.0,
                                          window=window)
                assert abs(float(out[-1].float().mean()) - (1.0 if j >= edge else 0.0)) < 1e-2, (window, i, j)


# ----------------------------------------------------------------------------------------------------- latent attention
def latent_rows(rank, rot, n, dtype, seed=1):
    rows = torch.zeros(n, ops.latent_width(rank + rot), dtype=dtype)
    rows[:, :rank + rot] = rand(n, rank + rot, seed=seed, dtype=dtype)
    return rows


def latent_pages(rows, bs, seed=0):
    kc, _, bt = paged(rows[:, None], rows[:, None], bs, seed)
    return kc[:, 0].contiguous(), bt


def latent_oracle(rows, q, uk, uv, scale, rank, rot, gate, window, sink):
    f, (n, H) = rows.float(), q.shape[:2]
    k = torch.cat([torch.einsum("tr,hnr->thn", f[:, :rank], uk.float()), f[:, None, rank:rank + rot].expand(-1, H, -1)], -1)
    v = torch.einsum("tr,hvr->thv", f[:, :rank], uv.float())
    o = O.attend(q.float(), k, v, scale, O.window_mask(n, window) if window else O.causal_mask(n), None, sink)
    return (o * O.sigmoid(gate.float())[:, :, None]).reshape(n, -1)


LATENT = pytest.mark.parametrize("H,N,rot,V,rank,window,bs", [
    (4, 24, 16, 40, 48, 45, 16), (36, 16, 16, 16, 200, 150, 16), (2, 128, 64, 128, 512, 64, 32), (16, 64, 64, 64, 128, 1, 64),
    (5, 12, 6, 20, 28, 31, 16), (33, 32, 8, 32, 136, 400, 8), (3, 16, 16, 16, 64, 0, 16)])


def latent_case(H, N, rot, V, rank, dtype, n=333):
    rows, q = latent_rows(rank, rot, n, dtype), rand(n, H, N + rot, seed=2, dtype=dtype)
    uk, uv = (rand(H, d, rank, seed=s, dtype=dtype, scale=rank ** -0.5) for d, s in ((N, 3), (V, 4)))
    return rows, q, uk, uv, rand(n, H, seed=5, dtype=dtype, scale=2.0), rand(H, seed=6, scale=3.0)


@DTYPES
@pytest.mark.parametrize("impl", ["tc", "simt"])
@LATENT
def test_latent_attention_in_the_latent_space(dtype, impl, H, N, rot, V, rank, window, bs):
    if impl == "tc" and (dtype == F32 or N % 8):
        pytest.skip("the tensor-core kernels are bf16, with sizes in multiples of 8")
    scale = 0.25
    rows, q, uk, uv, gate, sink = latent_case(H, N, rot, V, rank, dtype)
    want = latent_oracle(rows, q, uk, uv, scale, rank, rot, gate, window, sink)
    pages, bt = latent_pages(rows, bs)
    for lo, hi in ((0, 1), (127, 129), (250, 282), (332, 333), (255, 257)):
        T = hi - lo
        qa = ops.latent_queries(q[lo:hi].cuda(), uk.cuda(), impl=impl)
        for max_ctx in (hi, 20000):  # another number of splits
            lat = ops.latent_attention(qa, pages, bt, i32(0, T), i32(hi), rank, scale=scale, max_ctx=max_ctx, window=window,
                                       sink=sink.cuda(), impl=impl)
            out = torch.empty(T, H * V, dtype=dtype, device="cuda")
            ops.latent_values(lat, uv.cuda(), gate[lo:hi].cuda(), out, impl=impl)
            close(out, want[lo:hi], dtype, bf16=2e-2)


@LATENT
def test_latent_attention_expanded(H, N, rot, V, rank, window, bs):
    """Two sequences over the same pages, their contexts cut to what the window reaches from the first query."""
    if not ops.latent_prefill_supported(H, N, rot, V, rank, BF, "cuda"):
        assert N % 8 or rot % 8
        return
    n, scale = 333, 0.25
    rows, q, uk, uv, gate, sink = latent_case(H, N, rot, V, rank, BF)
    want = latent_oracle(rows, q, uk, uv, scale, rank, rot, gate, window, sink)
    pages, bt = latent_pages(rows, bs)
    up = torch.cat([uk.reshape(-1, rank), uv.reshape(-1, rank)]).cuda()
    lo, hi = 150, 290
    c2 = min(hi, hi - lo + window - 1) if window else hi
    ctx = i32(0, n, n + c2)
    got_rows = ops.latent_gather(pages, torch.cat([bt, bt]), ctx, n + c2, i32(n, hi))
    assert torch.equal(got_rows.cpu(), torch.cat([rows, rows[hi - c2:hi]]))
    kv = ops.gemm(got_rows[:, :rank], up)
    qq, gg = torch.cat([q, q[lo:hi]]).cuda(), torch.cat([gate, gate[lo:hi]]).cuda()
    out = torch.full((n + hi - lo + 3, H * V), 7.0, dtype=BF, device="cuda")
    ops.latent_prefill(qq, got_rows[:, rank:rank + rot], kv, i32(0, n, n + hi - lo), ctx, n, N, V, scale=scale, gate=gg, out=out,
                       window=window, sink=sink.cuda())
    close(out[:n], want, BF, bf16=2e-2)
    close(out[n:-3], want[lo:hi], BF, bf16=2e-2)
    assert bool((out[-3:] == 7.0).all())


@pytest.mark.parametrize("form", ["latent", "expanded"])
def test_latent_window_edges(form):
    """One key that outweighs all others just inside and just outside of the window."""
    H, N, rot, V, rank = 2, 16, 16, 16, 64
    uk, uv = torch.zeros(H, N, rank, dtype=BF).cuda(), torch.zeros(H, V, rank, dtype=BF).cuda()
    uv[:, :, 5] = 1.0
    for window, i in ((64, 63), (64, 64), (64, 700), (65, 128), (112, 111), (112, 112), (112, 300), (300, 640), (1, 130)):
        n, edge = i + 1, i - window + 1
        for j in {0, 1, edge - 1, edge, edge + 1, i - 1, i, i // 64 * 64, i // 64 * 64 - 1}:
            if not 0 <= j <= i:
                continue
            rows = torch.zeros(n, ops.latent_width(rank + rot), dtype=BF)
            rows[j, rank + 3], rows[j, 5] = 6.0, 1.0  # the rotated part stands out, the latent carries the value
            q = torch.zeros(n, H, N + rot, dtype=BF)
            q[:, :, N + 3] = 5.0
            pages, bt = latent_pages(rows, 16)
            if form == "latent":
                lat = ops.latent_attention(ops.latent_queries(q[-1:].cuda(), uk), pages, bt, i32(0, 1), i32(n), rank, scale=1.0,
                                           max_ctx=n, window=window)
                out = ops.latent_values(lat, uv, None, torch.empty(1, H * V, dtype=BF, device="cuda"))
            else:
                new = min(n, 3)
                c = min(n, new + window - 1)
                r = ops.latent_gather(pages, bt, i32(0, c), c, i32(n))
                kv = ops.gemm(r[:, :rank], torch.cat([uk.view(-1, rank), uv.view(-1, rank)]))
                out = torch.empty(new, H * V, dtype=BF, device="cuda")
                ops.latent_prefill(q[-new:].cuda(), r[:, rank:rank + rot], kv, i32(0, new), i32(0, c), new, N, V, scale=1.0, gate=None,
                                   out=out, window=window)
            assert abs(float(out[-1].float().mean()) - (1.0 if j >= edge else 0.0)) < 1e-2, (window, i, j)
    assert _lib.read_status()[0] == 0


@pytest.mark.parametrize("form", ["latent", "expanded"])
def test_latent_sinks(form):
    """Sinks far below, among and far above the scores: they take their share of the denominator and give no value."""
    H, N, rot, V, rank, n = 4, 16, 16, 16, 64, 200
    rows, q, uk, uv, gate, _ = latent_case(H, N, rot, V, rank, BF, n=n)
    sink = torch.tensor([-300.0, 0.0, 4.0, 80.0])
    gate = torch.zeros_like(gate)
    want = latent_oracle(rows, q, uk, uv, 0.5, rank, rot, gate, 70, sink).view(n, H, V)
    pages, bt = latent_pages(rows, 16)
    if form == "latent":
        lo = n - 5
        lat = ops.latent_attention(ops.latent_queries(q[lo:].cuda(), uk.cuda()), pages, bt, i32(0, 5), i32(n), rank, scale=0.5,
                                   max_ctx=n, window=70, sink=sink.cuda())
        out = ops.latent_values(lat, uv.cuda(), gate[lo:].cuda(), torch.empty(5, H * V, dtype=BF, device="cuda"))
    else:
        lo = 0
        r = ops.latent_gather(pages, bt, i32(0, n), n, i32(n))
        kv = ops.gemm(r[:, :rank], torch.cat([uk.reshape(-1, rank), uv.reshape(-1, rank)]).cuda())
        out = torch.empty(n, H * V, dtype=BF, device="cuda")
        ops.latent_prefill(q.cuda(), r[:, rank:rank + rot], kv, i32(0, n), i32(0, n), n, N, V, scale=0.5, gate=gate.cuda(), out=out,
                           window=70, sink=sink.cuda())
    out = out.view(-1, H, V).float().cpu()
    for h in range(3):
        close(out[:, h], want[lo:, h], BF, bf16=2e-2)
    assert float(out[:, 3].abs().max()) < 1e-6 and float((want[:, 2] - want[:, 1]).abs().max()) > 1e-2


# ---------------------------------------------------------------------------------------------------- linear recurrent unit
def lru_weights(W, blocks, taps, dtype, seed=0):
    n = W // blocks
    return (rand(W, taps, seed=seed + 1, dtype=dtype, scale=taps ** -0.5), rand(W, seed=seed + 2, dtype=dtype, scale=0.3),
            rand(2 * blocks, n, n, seed=seed + 3, dtype=dtype, scale=2 * n ** -0.5), rand(2 * blocks, n, seed=seed + 4),
            torch.rand(W, generator=torch.Generator().manual_seed(seed + 5)) * 8 - 7)


def lru_oracle(proj, w, blocks, power=8.0):
    """One whole sequence: (output [T, W], states [T, W])."""
    conv, cb, gates, gb, lam = (t.float() for t in w)
    W = conv.shape[0]
    u = O.causal_conv(proj[:, W:2 * W].float(), conv, cb)
    u = u.to(proj.dtype).float()  # an activation
    r, i = (O.sigmoid(O.block_linear(u, gates[k * blocks:(k + 1) * blocks], gb[k * blocks:(k + 1) * blocks])) for k in range(2))
    S = O.linear_scan(*O.lru_gates(u, r, i, lam))
    return S * O.gelu_tanh(proj[:, :W].float()), S


LRU_SIZES = [(128, 1, 4), (144, 3, 4), (96, 12, 1), (272, 2, 3), (384, 1, 5), (60, 5, 3), (512, 2, 9), (320, 1, 2), (640, 5, 4)]


@DTYPES
@pytest.mark.parametrize("impl", ["tc", "split", "simt"])
@pytest.mark.parametrize("W,blocks,taps", LRU_SIZES)
def test_linear_recurrent_unit(dtype, impl, W, blocks, taps):
    """Unequal sequences in steps of portions and single tokens, in slots that others have used, against whole sequences."""
    n = W // blocks
    if impl != "simt" and (dtype == F32 or n % 8 or (impl == "tc" and n > 320)):
        pytest.skip("the tensor-core forms are bf16, blocks in multiples of 8, in the fused one up to 320")
    w = lru_weights(W, blocks, taps, dtype)
    dev = [t.cuda() for t in w]
    lens = [200, 70, 5, 131]
    seqs = [rand(L, 2 * W + 8, seed=10 + i, dtype=dtype) for i, L in enumerate(lens)]
    want = [lru_oracle(s, w, blocks) for s in seqs]
    ring, state = rand(6, taps, W, seed=20, dtype=dtype, scale=9.0).cuda(), rand(6, W, seed=21, scale=9.0).cuda()  # used slots
    slot, at = [4, 0, 5, 2], [0] * 4
    for step in ([(0, 64), (3, 1)], [(0, 1), (1, 2), (3, 65)], [(2, 1), (0, 1)], [(0, 70), (1, 66), (2, 2), (3, 1)],
                 [(0, 1), (1, 1), (2, 1), (3, 1)], [(3, 63), (0, 63), (1, 1), (2, 1)]):
        step = sorted(step, key=lambda e: e[1] > 1)
        c = [k for _, k in step]
        proj = torch.cat([seqs[s][at[s]:at[s] + k] for s, k in step])
        total = [at[s] + k for s, k in step]
        out = ops.rglru(proj.cuda(), *dev, ring, state, i32(*np.cumsum([0] + c).tolist()), i32(*total), i32(*[slot[s] for s, _ in step]),
                        max(c), singles=sum(k == 1 for k in c), impl=impl)
        lo = 0
        for s, k in step:
            close(out[lo:lo + k], want[s][0][at[s]:at[s] + k], dtype, bf16=4e-3)
            close(state[slot[s]], want[s][1][at[s] + k - 1], F32, f32=1e-4 if dtype == BF else 2e-5)
            lo, at[s] = lo + k, at[s] + k
    assert at == lens
    close(state[1], rand(6, W, seed=21, scale=9.0)[1], F32, f32=1e-9)  # nobody's slot


@DTYPES
@pytest.mark.parametrize("decode", [False, True])
def test_recurrence_remembers_from_far_away(dtype, decode):
    """Decays near one: the first token's input is still there a thousand tokens on, and nothing is lost from portion to
    portion. Tiny inputs against a large state: 16 bits would swallow them."""
    W, T = 64, 1200
    conv, cb = torch.zeros(W, 2, dtype=dtype), torch.zeros(W, dtype=dtype)
    conv[:, 1] = 1.0
    gates, gb = torch.zeros(8, 16, 16, dtype=dtype), torch.zeros(8, 16)
    lam = torch.full((W,), -9.0)
    proj = torch.zeros(T, 2 * W, dtype=dtype)
    proj[:, :W], proj[:, W:] = 3.0, 0.01
    proj[0, W:] = 500.0
    w = (conv, cb, gates, gb, lam)
    want, S = lru_oracle(proj, w, 4)
    assert float(S[-1].mean()) > 0.4 * float(S[0].mean())
    ring, state, out, at = torch.zeros(1, 2, W, dtype=dtype).cuda(), torch.zeros(1, W).cuda(), [], 0
    for k in [T - 300] + [1] * 300 if decode else [500, 2, 64, 63, T - 629]:
        out.append(ops.rglru(proj[at:at + k].cuda(), *[t.cuda() for t in w], ring, state, i32(0, k), i32(at + k), i32(0), k))
        at += k
    close(torch.cat(out), want, dtype, bf16=4e-3, f32=5e-5)
    close(state[0], S[-1], F32, f32=1e-4)


def test_recurrence_extreme_gates():
    """Gates at both ends, gelu of large numbers: finite, as the equations say."""
    W, T = 128, 80
    proj, w = rand(T, 2 * W, seed=1, dtype=BF, scale=30.0), list(lru_weights(W, 2, 3, BF))
    w[3] = w[3] * 60
    want, _ = lru_oracle(proj, w, 2)
    args = [t.cuda() for t in w]
    for sizes in ([T], [1] * T):
        ring, state, out, at = torch.zeros(1, 3, W, dtype=BF).cuda(), torch.zeros(1, W).cuda(), [], 0
        for k in sizes:
            out.append(ops.rglru(proj[at:at + k].cuda(), *args, ring, state, i32(0, k), i32(at + k), i32(0), k))
            at += k
        out = torch.cat(out)
        assert bool(torch.isfinite(out).all())
        close(out, want, BF, bf16=4e-3)


# ----------------------------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("T", [1, 7, 32, 33, 500, 5000])
@pytest.mark.parametrize("E,top", [(1, 1), (5, 2), (16, 1), (40, 5), (130, 8), (300, 32), (512, 3)])
def test_routing(T, E, top):
    z = rand(T, E + 3, seed=T, scale=2.0)
    z[0, :min(E, 4)] = 40.0  # saturated scores: equal, the lower expert first
    counters = torch.zeros(E + 1, dtype=torch.int32).cuda()
    for score, norm in (("sigmoid", False), ("softmax", True)):
        r = ops.moe_route(z.cuda(), E, top, counters, score=score, renormalize=norm)
        s = torch.sigmoid(z[:, :E]) if score == "sigmoid" else torch.softmax(z[:, :E], -1)
        idx = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :top]
        w = s.gather(1, r.idx.cpu().long())
        close(r.weight, w / w.sum(-1, keepdim=True) if norm else w, F32, f32=1e-5)
        clear = torch.ones(T, dtype=torch.bool)  # but for scores that are equal to the last bits
        v = s.sort(-1, descending=True).values
        if E > 1:
            clear = ((v[:, :-1] - v[:, 1:])[:, :top] > 1e-6).all(1)
        assert torch.equal(r.idx.cpu().long()[clear], idx[clear])
        if score == "sigmoid":
            assert r.idx[0].tolist() == idx[0].tolist()[:top] or top > 4
        dest, e = r.dest.cpu().flatten().long(), r.idx.cpu().flatten().long()
        assert len(set(dest.tolist())) == T * top and torch.equal(r.blk_expert.cpu().long()[dest // 128], e)
        used = (torch.bincount(e, minlength=E) + 127).div(128, rounding_mode="floor").sum()
        assert int((r.blk_expert >= 0).sum()) == int(used) and int(counters.abs().sum()) == 0


@DTYPES
@pytest.mark.parametrize("weigh", ["input", "output"])
@pytest.mark.parametrize("T,H,E,top,ff,shared", [(1, 64, 4, 2, 48, 40), (37, 96, 5, 3, 64, 0), (300, 136, 8, 1, 72, 136),
                                                 (700, 52, 3, 2, 44, 20), (130, 256, 12, 4, 200, 64)])
def test_experts_and_their_sum(dtype, weigh, T, H, E, top, ff, shared):
    x, logits = rand(T, H, seed=1, dtype=dtype), rand(T, E + 1, seed=2, scale=2.0)
    gu, down = rand(E, 2 * ff, H, seed=3, dtype=dtype, scale=2 * H ** -0.5), rand(E, H, ff, seed=4, dtype=dtype, scale=ff ** -0.5)
    sh, res, nw = rand(T, H + 8, seed=5, dtype=dtype)[:, :H], rand(T, H, seed=6, scale=2.0), rand(H, seed=7, dtype=dtype)
    idx, wt = O.route(logits[:, :E], torch.eye(E), top)
    want = res.clone()
    for e in range(E):
        t, k = (idx == e).nonzero(as_tuple=True)
        w = {"gate": gu[e, :ff].float(), "up": gu[e, ff:].float(), "down": down[e].float()}
        c = wt[t, k][:, None]
        want[t] += O.glu(x[t].float(), w.get, "", c) if weigh == "input" else O.glu(x[t].float(), w.get, "") * c
    if shared:
        want += sh.float() * O.sigmoid(logits[:, E:])
    counters = torch.zeros(E + 1, dtype=torch.int32).cuda()
    lg = logits.cuda()
    r = ops.moe_route(lg, E, top, counters)
    out = ops.moe_experts(x.cuda(), r, gu.cuda(), down.cuda(), "silu", weigh_input=weigh == "input")
    for norm in (None, nw):
        got = res.cuda()
        parts = ops.RoutedSum(out, r, weigh == "output", sh.cuda() if shared else None, lg[:, E] if shared else None)
        y = ops.moe_combine(parts, got, None if norm is None else norm.cuda(), 1e-3)
        close(got, want, dtype)
        close(y, want if norm is None else O.rms_norm(want, 1e-3, norm.float()), dtype)


def test_experts_do_not_depend_on_company():
    """A token's result does not depend on who else is in the step."""
    H, E, ff = 128, 6, 64
    x, z = rand(400, H, seed=1, dtype=BF).cuda(), rand(400, E, seed=2, scale=2.0).cuda()
    gu, down = rand(E, 2 * ff, H, seed=3, dtype=BF, scale=0.1).cuda(), rand(E, H, ff, seed=4, dtype=BF, scale=0.1).cuda()
    c = torch.zeros(E + 1, dtype=torch.int32).cuda()

    def run(lo, hi):
        r = ops.moe_route(z[lo:hi], E, 2, c)
        out = moe_ops.moe_experts(x[lo:hi], r, gu, down, "silu", weigh_input=True)
        res = torch.zeros(hi - lo, H, device="cuda")
        ops.moe_combine(ops.RoutedSum(out, r, False), res, None, 0.0)
        return res

    whole = run(0, 400)
    for lo, hi in ((0, 1), (17, 60), (399, 400)):
        assert torch.equal(run(lo, hi), whole[lo:hi])


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


def test_routers_that_read_the_whole_stream(tmp_path):
    """fp32, where close calls are rare enough: routers without prepared choices."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=8, clear=False)
    eng = M.engine(M.load_model(cfg, w, tmp_path, F32, "cuda"))
    ids = tokens(120, cfg["vocab"], 4)
    assert M.error(M.feed_portions(eng, "a", ids, [70, 1]), O.forward(cfg, w, ids)) < TOL[F32]


@DTYPES
def test_long_decoding(dtype, tmp_path):
    """Hundreds of decoded tokens: windows pass over decoded positions, pages are added one by one, the state goes on."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=6)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"))
    ids = tokens(500, cfg["vocab"], 1)
    assert M.error(M.feed_portions(eng, "a", ids, [3] + [1] * 497), O.forward(cfg, w, ids)) < TOL[dtype]


@DTYPES
@pytest.mark.parametrize("short", [1, 32])
def test_unequal_batches(dtype, short, tmp_path):
    """Portions beside single tokens (both forms of latent attention and of the recurrence in one step), requests that pause,
    pages and slots that change hands: each as if alone."""
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


@pytest.mark.parametrize("kw", [{}, {"enforce_eager": True, "decode_burst": 1}, {"max_num_batched_tokens": 32}, {"num_blocks": 10}])
def test_greedy_generation(kw, tmp_path):
    """generate() with its scheduler: CUDA graphs and bursts, eager steps, portions of prompts, preemption."""
    cfg = M.config([M.rglru(64, 2, 3, M.moe(4, 2, 32, 32)), M.latent(2, 16, 16, 32, 32, 24, 19),
                    M.attention(2, 1, 32, 23, mlp=M.moe(3, 1, 64, 16))], vocab=64, width=64, side=8)
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


def test_fp8_weights(tmp_path):
    """rollout.quantization = fp8: coarse, but the same model."""
    cfg = M.config([M.rglru(128, 2, 4, M.moe(4, 2, 64, 128)), M.latent(2, 64, 64, 64, 128, 128, 40),
                    M.attention(2, 1, 64, 40, mlp=M.moe(3, 1, 64, 128))], vocab=256, width=128)
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
