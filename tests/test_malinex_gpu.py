"""The Malinex design on the GPU: every mechanism's kernels alone, then whole models through the engine, against the plain
implementation in ``_malinex_oracle.py`` (on the CPU)."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import _malinex_models as M
import _malinex_oracle as O
from verl_b200 import ops
from verl_b200.ops import _lib
from verl_b200.ops.nn import activation
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
@pytest.mark.parametrize("H", [8, 52, 104, 4096])
def test_learned_positions(dtype, H):
    table, pos = rand(50, H, seed=4, dtype=dtype), rand(31, H, seed=5, dtype=dtype)
    ids, at = torch.tensor([0, 49, 7, 7, 3]), torch.tensor([0, 30, 5, 6, 29])
    got = ops.embedding_scaled(ids.cuda(), table.cuda(), 1.0, pos_table=pos.cuda(), positions=at.cuda())
    close(got, table.float()[ids] + pos.float()[at], F32)


@DTYPES
@pytest.mark.parametrize("H,pad", [(8, 0), (52, 3), (104, 8), (96, 4), (4096, 0)])
def test_gated_norm_and_add(dtype, H, pad):
    """The gate in rows of its own or behind other columns, aligned or not."""
    res, d, w, fw = rand(33, H, seed=1, scale=3.0), rand(33, H, seed=2, dtype=dtype), rand(H, seed=3, dtype=dtype), rand(H, seed=4, dtype=dtype)
    gate = rand(33, H + pad, seed=5, dtype=dtype, scale=2.0)[:, pad:]
    for g in (None, gate):
        y = d.float() * (1.0 if g is None else O.sigmoid(g.float()))
        want = res + O.rms_norm(y, 1e-2, w.float())
        for final in (None, fw):
            r = res.cuda()
            out = ops.rmsnorm_add(d.cuda(), r, w.cuda(), 1e-2, final_weight=None if final is None else final.cuda(), final_scale=0.7,
                                  gate=None if g is None else gate.cuda())
            close(r, want, F32, f32=2e-5 if dtype == F32 else 1e-3)
            close(out, want if final is None else O.rms_norm(want, 1e-2, fw.float()) * 0.7, dtype)


@DTYPES
@pytest.mark.parametrize("n", [64, 52, 37, 1024])
def test_activations(dtype, n):
    x = rand(256, n + 8, seed=5, dtype=dtype, scale=2.0)
    for act, f in (("gelu", O.gelu), ("relu2", O.relu2)):
        close(activation(x.cuda(), n, act), f(x[:, :n].float()), dtype, bf16=4e-3)
        got = activation(x.cuda(), n, act, i32(-1, 3))
        close(got[128:], f(x[128:, :n].float()), dtype, bf16=4e-3)
    with pytest.raises(ValueError):
        activation(x.cuda(), n, "tanh")


@DTYPES
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 32, 24), (3, 3, 20, 12), (8, 1, 128, 128), (2, 1, 144, 160)])
@pytest.mark.parametrize("temp", [None, (0.4, 30.0), (1.5, 1.0), (-0.2, 7.5)])
def test_projection_norm_and_query_temperature(dtype, H, G, D, V, temp):
    """Positions right before and after a step of the temperature, and far away."""
    BS, at = 16, torch.tensor([0, 1, 5, 6, 7, 13, 14, 28, 29, 30, 58, 59, 60, 899, 100000])
    T, nq, nk, nv = len(at), H * D, G * D, G * V
    x = rand(T, (nq + nk + nv + 15) // 8 * 8, seed=1, dtype=dtype)
    qw, kw = rand(nq, seed=2, dtype=dtype), rand(nk, seed=3, dtype=dtype)
    for norm in (True, False):
        kc, vc = torch.zeros(5, G, BS, D, dtype=dtype).cuda(), torch.zeros(5, G, BS, V, dtype=dtype).cuda()
        slots = torch.randperm(5 * BS, generator=torch.Generator().manual_seed(1))[:T]
        slots[3] = -1
        w = (qw.cuda(), kw.cuda()) if norm else (None, None)
        got = ops.qk_norm_kv_write(x.clone().cuda(), *w, slots.cuda(), kc, vc, H, 1e-2, q_temp=temp, positions=at.cuda())
        f = x.float()
        q, k = f[:, :nq], f[:, nq:nq + nk]
        if norm:
            q, k = O.rms_norm(q, 1e-2, qw.float()), O.rms_norm(k, 1e-2, kw.float())
        factor = O.query_temperature(at.tolist(), None if temp is None else {"coef": temp[0], "every": temp[1]}).float()
        close(got, (q * factor[:, None]).view(T, H, D), dtype)
        for t in range(T):  # each row on its own: a step missed at one position shows
            close(got[t], (q[t] * factor[t]).view(H, D), dtype)
        ok = slots >= 0
        blk, off = slots[ok] // BS, slots[ok] % BS
        close(kc.cpu()[blk, :, off], k.view(T, G, D)[ok], dtype)
        assert torch.equal(vc.cpu()[blk, :, off].reshape(-1, nv), x[:, nq + nk:nq + nk + nv][ok])


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
@pytest.mark.parametrize("biased", [True, False])
@pytest.mark.parametrize("H,G,D,V,bs", [(6, 3, 32, 24, 16), (8, 1, 64, 64, 8), (16, 1, 16, 40, 16), (4, 4, 128, 128, 128),
                                        (3, 3, 20, 12, 16), (2, 1, 144, 160, 32), (4, 2, 8, 128, 16)])
def test_sigmoid_attention(dtype, biased, H, G, D, V, bs):
    """Whole prompts, portions anywhere and single tokens; gate per head or none."""
    n = 333
    q, k, v = (rand(n, h, d, seed=s, dtype=dtype) for h, d, s in ((H, D, 1), (G, D, 2), (G, V, 3)))
    r1, r2 = rand(H, seed=4).abs() * 2, rand(H, seed=5).abs() + 0.1
    r1[0] = 0.0
    shift, gate = rand(H, seed=6) - 2.5, rand(n, H + 5, seed=7, dtype=dtype)[:, 5:]
    bias = O.distance_bias(n, r1, r2) if biased else torch.zeros(H, n, n)
    raw = O.sigmoid_attend(q.float(), k.float(), v.float(), 0.4, bias, shift)
    kc, vc, bt = paged(k, v, bs)
    dev = dict(scale=0.4, shift=shift.cuda(), log_bias=(r1.cuda(), r2.cuda()) if biased else None)
    for lo, hi in ((0, n), (0, 1), (127, 129), (200, 333), (332, 333), (128, 129), (130, 132)):
        for g in (None, gate):
            want = raw if g is None else raw * O.sigmoid(g.float())[:, :, None]
            got = ops.paged_attention(q[lo:hi].cuda(), kc, vc, bt, i32(0, hi - lo), i32(hi), hi - lo, **dev,
                                      gate=None if g is None else gate[lo:hi].cuda())
            close(got, want.reshape(n, -1)[lo:hi], dtype)


@DTYPES
def test_sigmoid_attention_of_long_sequences(dtype):
    """Many blocks of keys, a step's keys split over CTAs, unequal sequences in one step."""
    H, G, D = 4, 2, 64
    lens, new = [2100, 700, 130, 1], [140, 3, 128, 1]
    dev = [t.cuda() for t in (rand(H, seed=4).abs(), rand(H, seed=5).abs() + 0.1, rand(H, seed=6) - 4)]
    cpu = [t.cpu() for t in dev]
    qs, kcs, vcs, tables, wants, base = [], [], [], [], [], 0
    for b, n in enumerate(lens):
        q, k, v = (rand(n, h, D, seed=10 * b + s, dtype=dtype) for h, s in ((H, 1), (G, 2), (G, 3)))
        wants.append(O.sigmoid_attend(q.float(), k.float(), v.float(), 0.2, O.distance_bias(n, *cpu[:2]), cpu[2]).reshape(n, -1))
        kc, vc, bt = paged(k, v, 16, b)
        qs.append(q)
        kcs.append(kc)
        vcs.append(vc)
        tables.append(bt[0] + base)
        base += kc.shape[0]
    table = torch.zeros(4, max(len(t) for t in tables), dtype=torch.int32).cuda()
    for b, t in enumerate(tables):
        table[b, :len(t)] = t
    kc, vc = torch.cat(kcs), torch.cat(vcs)
    opts = dict(scale=0.2, shift=dev[2], log_bias=(dev[0], dev[1]), max_ctx=2100)
    for counts in (new, [1] * 4):
        q = torch.cat([x[len(x) - c:] for x, c in zip(qs, counts)]).cuda()
        got = ops.paged_attention(q, kc, vc, table, i32(*np.cumsum([0] + counts).tolist()), i32(*lens), max(counts), **opts)
        lo = 0
        for w, c in zip(wants, counts):  # single queries have small sums of small weights: each sequence on its own
            close(got[lo:lo + c], w[len(w) - c:], dtype, bf16=1.5e-2)
            lo += c


@DTYPES
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_far_away(dtype, decode):
    """All other weights vanish: the output is the value of the one key that scores, at page and block borders and at the first
    token, times the sigmoid of what the distance leaves of the score; a key that comes later than the query adds nothing."""
    D, bs, shift, r1, r2 = 32, 16, -30.0, 1.3, 0.4
    dev = dict(scale=1.0, shift=torch.tensor([shift]).cuda(), log_bias=(torch.tensor([r1]).cuda(), torch.tensor([r2]).cuda()))
    for i in (0, 1, 15, 16, 127, 128, 129, 300, 511):
        for j in {0, 1, 15, 16, i - 1, i, i + 1, i + 2, 127, 128, i // 16 * 16, i // 16 * 16 - 1, i // 128 * 128}:
            if j < 0:
                continue
            n = max(i, j) + 1
            q, k, v = torch.zeros(n, 1, D), torch.zeros(n, 1, D), torch.zeros(n, 1, D)
            q[:, 0, 3], k[j, 0, 3], v[j, 0] = 5.0, 7.0, 1.0
            kc, vc, bt = paged(k.to(dtype), v.to(dtype), bs)
            want = float(torch.sigmoid(torch.tensor(35 + shift - r1 * np.log1p(r2 * (i - j)), dtype=torch.float64))) if j <= i else 0.0
            lo = i if decode else max(0, i - 2)
            out = ops.paged_attention(q[lo:i + 1].to(dtype).cuda(), kc, vc, bt, i32(0, i + 1 - lo), i32(i + 1), i + 1 - lo, **dev)
            assert abs(float(out[-1].float().mean()) - want) < (1e-5 if dtype == F32 else 4e-3), (i, j)


def test_extreme_scores():
    """Scores of many thousands either way: weights of exactly zero and one, nothing overflows."""
    n, D = 200, 64
    q, k, v = (rand(n, 2, D, seed=s, dtype=BF, scale=100.0) for s in (1, 2, 3))
    shift, r = torch.tensor([-5.0, 800.0]), torch.tensor([0.5, 3.0])
    want = O.sigmoid_attend(q.double(), k.double(), v.double(), 1.0, O.distance_bias(n, r.double(), r.double()), shift.double())
    kc, vc, bt = paged(k, v, 16)
    dev = dict(scale=1.0, shift=shift.cuda(), log_bias=(r.cuda(), r.cuda()))
    close(ops.paged_attention(q.cuda(), kc, vc, bt, i32(0, n), i32(n), n, **dev), want.reshape(n, -1), BF)
    close(ops.paged_attention(q[-1:].cuda(), kc, vc, bt, i32(0, 1), i32(n), 1, **dev), want.reshape(n, -1)[-1:], BF)


def test_attention_refuses_mixed_forms():
    q = torch.zeros(1, 1, 16, device="cuda", dtype=BF)
    kc = torch.zeros(1, 1, 16, 16, device="cuda", dtype=BF)
    one = torch.zeros(1, device="cuda")
    args = (q, kc, kc, i32(0).view(1, 1), i32(0, 1), i32(1), 1)
    for kw in (dict(shift=one, sink=one), dict(shift=one, softcap=3.0), dict(log_bias=(one, one)),
               dict(gate=torch.zeros(1, 3, device="cuda", dtype=BF))):
        with pytest.raises(ValueError):
            ops.paged_attention(*args, scale=1.0, **kw)


# --------------------------------------------------------------------------------------------- gated linear attention
def gla_weights(H, D, V, rank, dtype, seed=0, lo=-3.0, hi=6.0):
    b = torch.rand(H * D, generator=torch.Generator().manual_seed(seed + 1)) * (hi - lo) + lo
    return rand(H * D, rank, seed=seed, dtype=dtype, scale=rank ** -0.5), b, rand(V, seed=seed + 2, dtype=dtype)


def gla_oracle(proj, w, H, D, V, tau, eps, keep=()):
    """Output [T, H V] and the states [H, D, V] behind the token counts in ``keep``, in double precision."""
    T, R = proj.shape[0], w[0].shape[1]
    x = proj.double()
    q, k, v, g, r = x[:, :2 * H * (D + V) + R].split([H * D, H * D, H * V, H * V, R], 1)
    a = O.decays(r @ w[0].double().T + w[1].double(), tau).view(T, H, D)
    q, k, v = q.reshape(T, H, D) * D ** -0.5, k.reshape(T, H, D), v.reshape(T, H, V)
    S, out, states = None, [], {}
    at = 0
    for t in sorted(set(keep) | {T}):
        o, S = O.linear_attention(q[at:t], k[at:t], v[at:t], a[at:t], S)
        out.append(o)
        states[t], at = S, t
    o = O.rms_norm(torch.cat(out), eps, w[2].double()).reshape(T, H * V)
    return o * O.silu(g), states


GLA_SIZES = [(3, 24, 40, 8, 5.0), (2, 128, 128, 16, 16.0), (1, 64, 64, 64, 1.0), (4, 32, 32, 5, 8.0), (2, 8, 136, 24, 2.0), (1, 72, 256, 12, 30.0),
             (5, 12, 20, 3, 3.0), (2, 7, 9, 6, 4.0), (1, 160, 136, 8, 7.0), (1, 16, 8, 80, 7.0)]


@DTYPES
@pytest.mark.parametrize("impl", ["chunk", "scan"])
@pytest.mark.parametrize("H,D,V,rank,tau", GLA_SIZES)
def test_gated_linear_attention(dtype, impl, H, D, V, rank, tau):
    """Unequal sequences in steps of portions and single tokens, in slots that others have used, against whole sequences."""
    if impl == "chunk" and (dtype == F32 or D % 8 or V % 8 or D > 128 or rank > 64):
        pytest.skip("the chunked form is bf16, sizes in multiples of 8")
    w = gla_weights(H, D, V, rank, dtype)
    dev = [t.cuda() for t in w]
    lens = [200, 70, 5, 131]
    steps = ([(0, 64), (3, 1)], [(0, 1), (1, 2), (3, 65)], [(2, 1), (0, 1)], [(0, 70), (1, 66), (2, 2), (3, 1)],
             [(0, 1), (1, 1), (2, 1), (3, 1)], [(3, 63), (0, 63), (1, 1), (2, 1)])
    seqs = [rand(L, (2 * H * (D + V) + rank + 15) // 8 * 8, seed=10 + i, dtype=dtype) for i, L in enumerate(lens)]
    ends = {s: set() for s in range(4)}
    at = [0] * 4
    for step in steps:
        for s, k in step:
            at[s] += k
            ends[s].add(at[s])
    assert at == lens
    want = [gla_oracle(x, w, H, D, V, tau, 1e-3, ends[s]) for s, x in enumerate(seqs)]
    used = rand(6, H, V, D, seed=21, scale=9.0)
    state = used.cuda()  # used slots
    slot, at = [4, 0, 5, 2], [0] * 4
    for step in steps:
        step = sorted(step, key=lambda e: e[1] > 1)
        c = [k for _, k in step]
        proj = torch.cat([seqs[s][at[s]:at[s] + k] for s, k in step])
        total = [at[s] + k for s, k in step]
        out = ops.gated_linear_attention(proj.cuda(), *dev, state, i32(*np.cumsum([0] + c).tolist()), i32(*total),
                                         i32(*[slot[s] for s, _ in step]), max(c), H, D, V, tau, 1e-3,
                                         singles=sum(k == 1 for k in c), impl=impl if max(c) > 1 else "auto")
        lo = 0
        for s, k in step:
            close(out[lo:lo + k], want[s][0][at[s]:at[s] + k], dtype, bf16=6e-3)
            close(state[slot[s]].transpose(1, 2), want[s][1][at[s] + k], F32, f32=1e-4 if dtype == BF else 2e-5)
            lo, at[s] = lo + k, at[s] + k
    for s in (1, 3):
        assert torch.equal(state[s].cpu(), used[s])  # nobody's slots


@DTYPES
@pytest.mark.parametrize("sizes", [[1200], [900] + [1] * 300, [500, 2, 64, 63, 571]])
def test_state_remembers_from_far_away(dtype, sizes):
    """Decays near one: the first token's large value is still there a thousand tokens on, and nothing is lost from portion to
    portion. Small values against a large state: 16 bits would swallow them."""
    H, D, V, T = 2, 64, 32, 1200
    w = (torch.zeros(H * D, 8, dtype=dtype), torch.full((H * D,), 7.0), torch.ones(V, dtype=dtype))
    proj = rand(T, 2 * H * (D + V) + 8, seed=1, dtype=dtype)
    proj[:, :2 * H * D] = proj[:, :2 * H * D].abs()
    proj[:, 2 * H * D:2 * H * D + H * V] *= 0.01
    proj[0, 2 * H * D:2 * H * D + H * V] *= 5e4
    want, S = gla_oracle(proj, w, H, D, V, 4.0, 1e-6, [1])
    assert float(S[T].abs().mean()) > 0.5 * float(S[1].abs().mean())
    state, out, at = torch.zeros(1, H, V, D).cuda(), [], 0
    for k in sizes:
        out.append(ops.gated_linear_attention(proj[at:at + k].cuda(), *[t.cuda() for t in w], state, i32(0, k), i32(at + k), i32(0), k,
                                              H, D, V, 4.0, 1e-6))
        at += k
    close(torch.cat(out), want, dtype, bf16=6e-3, f32=5e-5)
    close(state[0].transpose(1, 2), S[T], F32, f32=1e-4)


@pytest.mark.parametrize("case", ["strong", "one_channel", "bursts", "endless"])
@pytest.mark.parametrize("D,V", [(64, 64), (128, 24)])
def test_decays_of_any_strength(case, D, V):
    """Chunks in which e^-b leaves fp32's range for some channel are taken in pieces: strong decays everywhere, in one channel
    only, in single tokens between lasting ones (what a piece keeps must not suffer), and decays beyond all numbers."""
    H, T, tau = 2, 300, 1.0
    proj = rand(T, 2 * H * (D + V) + 8, seed=1, dtype=BF)
    r = proj[:, 2 * H * (D + V):]
    w0, b = torch.zeros(H * D, 8, dtype=BF), torch.full((H * D,), 8.0)
    r[:] = 0
    r[:, 0] = 1.0
    if case == "strong":
        b = torch.linspace(-12, 9, H * D)
    elif case == "one_channel":
        b[3] = -9.0
    elif case == "bursts":
        w0[:, 1] = torch.linspace(-1.0, 0.0, H * D).to(BF)
        r[::37, 1] = 60.0
        r[100:140, 1] = 25.0
    else:
        w0[:, 1] = -1.0
        r[50:60, 1] = 3e38
        r[200, 1] = 1e4
    w = (w0, b, torch.ones(V, dtype=BF))
    want, S = gla_oracle(proj, w, H, D, V, tau, 1e-3)
    for sizes in ([T], [70, 2, 64, 64, 100], [1] * T):
        state, out, at = torch.zeros(1, H, V, D).cuda(), [], 0
        for k in sizes:
            out.append(ops.gated_linear_attention(proj[at:at + k].cuda(), *[t.cuda() for t in w], state, i32(0, k), i32(at + k), i32(0),
                                                  k, H, D, V, tau, 1e-3))
            at += k
        out = torch.cat(out)
        assert bool(torch.isfinite(out).all()) and _lib.read_status()[0] == 0
        for lo in range(0, T, 20):
            close(out[lo:lo + 20], want[lo:lo + 20], BF, bf16=8e-3)
        close(state[0].transpose(1, 2), S[T], F32, f32=1e-4)


# ----------------------------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("T", [1, 7, 32, 33, 500, 5000])
@pytest.mark.parametrize("E,top", [(1, 1), (5, 2), (16, 1), (40, 5), (130, 8), (300, 32), (512, 3), (6, 6)])
def test_corrected_routing(T, E, top):
    """Chosen by score plus correction, weighted by the scores alone."""
    z, corr = rand(T, E + 3, seed=T, scale=2.0), torch.rand(E, generator=torch.Generator().manual_seed(E)) * 2 - 1
    corr[:: 3] = 0.0
    counters = torch.zeros(E + 1, dtype=torch.int32).cuda()
    r = ops.moe_route(z.cuda(), E, top, counters, score="softmax", renormalize=True, correction=corr.cuda())
    s = torch.softmax(z[:, :E].double(), -1)
    v, idx = (s + corr.double()).sort(-1, descending=True)
    w = s.gather(1, r.idx.cpu().long())
    close(r.weight, w / w.sum(-1, keepdim=True), F32, f32=1e-5)
    clear = ((v[:, :-1] - v[:, 1:])[:, :top] > 1e-6).all(1) if E > 1 else torch.ones(T, dtype=torch.bool)
    assert torch.equal(r.idx.cpu().long()[clear], idx[clear, :top])
    dest, e = r.dest.cpu().flatten().long(), r.idx.cpu().flatten().long()
    assert len(set(dest.tolist())) == T * top and torch.equal(r.blk_expert.cpu().long()[dest // 128], e)
    assert int(counters.abs().sum()) == 0


def test_vanishing_scores_of_the_chosen():
    """A correction may choose experts whose scores round to zero: shares stay finite."""
    z, E = torch.zeros(3, 8), 6
    z[:, 5] = 300.0
    corr = torch.tensor([9.0, 9.0, 0, 0, 0, -9.0])
    r = ops.moe_route(z.cuda(), E, 2, torch.zeros(E + 1, dtype=torch.int32).cuda(), score="softmax", renormalize=True,
                      correction=corr.cuda())
    assert r.idx.tolist() == [[0, 1]] * 3 and float(r.weight.abs().sum()) == 0


@DTYPES
@pytest.mark.parametrize("act", ["relu2", "gelu"])
@pytest.mark.parametrize("T,H,E,top,ff,shared", [(1, 64, 4, 2, 48, True), (37, 96, 5, 3, 64, False), (300, 136, 8, 1, 72, True),
                                                 (700, 52, 3, 2, 44, True), (130, 256, 12, 4, 200, False)])
def test_plain_experts_and_their_gated_normed_sum(dtype, act, T, H, E, top, ff, shared):
    x, logits, corr = rand(T, H, seed=1, dtype=dtype), rand(T, E, seed=2, scale=2.0), rand(E, seed=8)
    up, down = rand(E, ff, H, seed=3, dtype=dtype, scale=2 * H ** -0.5), rand(E, H, ff, seed=4, dtype=dtype, scale=ff ** -0.5)
    sh, gate = rand(T, H + 8, seed=5, dtype=dtype)[:, :H], rand(T, H + 16, seed=9, dtype=dtype)[:, 16:]
    res, nw, fw = rand(T, H, seed=6, scale=2.0), rand(H, seed=7, dtype=dtype), rand(H, seed=10, dtype=dtype)
    idx, wt = O.route(logits, torch.eye(E), corr, top)
    d = sh.float().clone() if shared else torch.zeros(T, H)
    for e in range(E):
        t, k = (idx == e).nonzero(as_tuple=True)
        w = {"up": up[e].float(), "down": down[e].float()}
        d[t] += O.two_layers(x[t].float(), w.get, "", {"relu2": O.relu2, "gelu": O.gelu}[act]) * wt[t, k][:, None]
    r = ops.moe_route(logits.cuda(), E, top, torch.zeros(E + 1, dtype=torch.int32).cuda(), score="softmax", renormalize=True,
                      correction=corr.cuda())
    out = ops.moe_experts(x.cuda(), r, up.cuda(), down.cuda(), act, weigh_input=False)
    parts = ops.RoutedSum(out, r, True, sh.cuda() if shared else None)
    for g in (None, gate):
        want = res + O.rms_norm(d if g is None else d * O.sigmoid(g.float()), 1e-3, nw.float())
        for final in (None, fw):
            got = res.cuda()
            y = ops.moe_norm_add(parts, got, nw.cuda(), 1e-3, gate=None if g is None else gate.cuda(), final_scale=0.5,
                                 final_weight=None if final is None else fw.cuda())
            close(got, want, dtype)
            close(y, want if final is None else O.rms_norm(want, 1e-3, fw.float()) * 0.5, dtype)


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
    """Hundreds of decoded tokens up to the last learned position: pages are added one by one, the state goes on."""
    cfg = {**M.CONFIGS["mixed"], "max_positions": 500}
    w = M.weights(cfg, seed=6)
    eng = M.engine(M.load_model(cfg, w, tmp_path, dtype, "cuda"))
    ids = tokens(500, cfg["vocab"], 1)
    assert M.error(M.feed_portions(eng, "a", ids, [3] + [1] * 497, end=False), O.forward(cfg, w, ids)) < TOL[dtype]
    with pytest.raises(Exception, match="max_model_len"):
        eng.feed([("a", [1], [0])])


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
    """bf16: the same request alone and in batches differs by rounding only (below the error against fp32)."""
    cfg = M.CONFIGS["mixed"]
    eng = M.engine(M.load_model(cfg, M.weights(cfg, seed=2), tmp_path, BF, "cuda"))
    ids, other = tokens(100, cfg["vocab"], 1), tokens(220, cfg["vocab"], 2)
    alone = M.feed_portions(eng, "a", ids, [100])
    got = eng.feed([("x", other[:130], []), ("a", ids, list(range(100))), ("y", other[:2], [])], ["a"]).cpu()
    assert M.error(got, alone) < TOL[BF] / 2
    assert M.error(M.feed_portions(eng, "b", ids, [7]), alone) < TOL[BF]


def greedy(cfg, w, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("kw", [{}, {"enforce_eager": True, "decode_burst": 1}, {"max_num_batched_tokens": 32}, {"num_blocks": 10}])
def test_greedy_generation(kw, tmp_path):
    """generate() with its scheduler: CUDA graphs and bursts, eager steps, portions of prompts, preemption."""
    cfg = M.config([M.gla(2, 32, 16, 3.0, M.moe(4, 2, 32, 32)), M.attention(2, 1, 32, 16, (0.5, 9), mlp=M.dense(48)), 0], vocab=64, width=64,
                   positions=96)
    w = M.weights(cfg, seed=5)
    eng = M.engine(M.load_model(cfg, w, tmp_path, F32, "cuda"), max_model_len=200, **kw)
    assert eng.max_model_len == 96
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
    cfg = M.config([M.gla(2, 64, 64, 8.0, M.moe(4, 2, 64, 128)), M.attention(2, 1, 64, 64, mlp=M.dense(128))], vocab=256, width=128)
    w = M.weights(cfg, seed=5)
    eng = M.engine(M.load_model(cfg, w, tmp_path, BF, "cuda"), quantization="fp8")
    ids = tokens(100, 256)
    want = O.forward(cfg, w, ids)
    assert float((M.feed_portions(eng, "a", ids, [60, 1, 39]) - want).pow(2).mean().sqrt() / want.std()) < 0.5


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
