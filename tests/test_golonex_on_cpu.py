"""The Golonex design in the framework, without a GPU: configuration and registry, checkpoints, the plan of a step, the engine's
batching and states, and greedy generation, against the plain implementation in ``_golonex_oracle.py``."""

import json

import numpy as np
import pytest
import torch

import _golonex_models as M
import _golonex_oracle as O
from verl_b200 import ops
from verl_b200.models import CausalLM, ModelConfig, build_model, preset
from verl_b200.models.hf_io import load_hf_checkpoint, native_to_hf_state_dict, save_hf_checkpoint
from verl_b200.models.layer_specs import RotarySpec
from verl_b200.models.registry import ModelRegistry
from verl_b200.rollout import SamplingParams


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


# ------------------------------------------------------------------------------------------- the oracle against other forms
def test_oracle_convolution():
    x, k, b = rand(9, 5, seed=1), rand(5, 4, seed=2), rand(5, seed=3)
    want = torch.nn.functional.conv1d(x.T[None], k[:, None], b, padding=3, groups=5)[0, :, :9].T
    assert torch.allclose(O.causal_conv(x, k, b), want, atol=1e-5)
    assert torch.allclose(O.causal_conv(x[:2], k, b), want[:2], atol=1e-5)  # shorter than the taps


def test_oracle_block_linear_is_a_block_diagonal_matrix():
    x, w, b = rand(7, 12, seed=1), rand(3, 4, 4, seed=2), rand(3, 4, seed=3)
    assert torch.allclose(O.block_linear(x, w, b), x @ torch.block_diag(*w).T + b.reshape(-1), atol=1e-5)


def test_oracle_recurrence():
    """Closed form with constant decay; the input's factor keeps a stationary state's variance."""
    T, C = 12, 3
    a, b = torch.full((T, C), 0.9, dtype=torch.float64), rand(T, C, seed=1).double()
    S = O.linear_scan(a, b)
    assert torch.allclose(S[-1], sum(0.9 ** (T - 1 - t) * b[t] for t in range(T)))
    assert torch.allclose(O.linear_scan(a[5:], b[5:], S[4]), S[5:])
    u = torch.ones(1, C, dtype=torch.float64)
    lam = torch.tensor([-3.0, 0.0, 2.0], dtype=torch.float64)
    a, v = O.lru_gates(u, torch.ones_like(u), torch.ones_like(u), lam)
    assert torch.allclose(a, torch.exp(-8 * torch.nn.functional.softplus(lam))) and torch.allclose(a * a + v * v, u)


def test_oracle_routing_and_windows():
    idx, w = O.route(torch.eye(2), torch.tensor([[1.0, -1.0], [3.0, 0.0], [2.0, 5.0]]), 2)
    assert idx.tolist() == [[1, 2], [2, 1]] and torch.allclose(w, torch.sigmoid(torch.tensor([[3.0, 2.0], [5.0, 0.0]])))
    m = O.window_mask(6, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 3, 3, 3] and bool(m[5, 3]) and not bool(m[5, 2]) and not bool(m[2, 3])


# ------------------------------------------------------------------------------------- configuration, registry, checkpoints
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_config_and_checkpoint_round_trip(name, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg)
    mc, native = load_hf_checkpoint(M.save(cfg, w, tmp_path / "a"))
    assert mc.model_type == "golonex" and mc.is_layer_list and mc.tie_word_embeddings and mc.to_hf_dict() == cfg
    assert mc.has_recurrent_state == any(x["type"] == "rglru" for x in cfg["layers"])
    assert mc.num_parameters() == sum(t.numel() for t in w.values())
    back = native_to_hf_state_dict(mc, native)
    assert back.keys() == w.keys() and all(torch.equal(back[k], w[k]) for k in w)
    save_hf_checkpoint(mc, native, tmp_path / "b")
    mc2, native2 = load_hf_checkpoint(tmp_path / "b")
    assert mc2 == mc and all(torch.equal(native2[k], native[k]) for k in native)


def test_registry():
    assert ModelRegistry.family("Golonex") == "golonex"
    build = ModelRegistry.load_model_cls("Golonex")
    assert type(build(preset("tiny-golonex"), dtype=torch.float32)).__name__ == "HybridLM"


def test_bad_configurations_are_refused(tmp_path):
    def changed(layer, key, value, part="mixer"):
        cfg = json.loads(json.dumps(M.CONFIGS["mixed"]))
        cfg["layers"][layer][part][key] = value
        return cfg

    for cfg, why in ((changed(1, "kv_heads", 4), "multiple"), (changed(1, "vdim", 16), "values"), (changed(0, "blocks", 5), "multiple"),
                     (changed(2, "rot_dim", 8), "rotated"), (changed(0, "kind", "sparse", "mlp"), "kind"),
                     (changed(1, "router", {"experts": 3, "top": 4}, "mlp"), "experts")):
        with pytest.raises(ValueError, match=why):
            ModelConfig.from_hf_dict(cfg)
    for cfg in (changed(2, "q_rank", 40), changed(0, "width", 72)):
        with pytest.raises(ValueError, match="rows"):
            load_hf_checkpoint(M.save(cfg, M.weights(M.CONFIGS["mixed"]), tmp_path))


def test_rotation_scaling_is_optional():
    rot = M.CONFIGS["mixed"]["layers"][1]["mixer"]["rot"]
    spec = RotarySpec.from_dict(rot, True)
    freqs, factor = O.rotation(rot)
    assert spec.frequencies() == pytest.approx(freqs, rel=1e-12) and spec.amplitude == pytest.approx(factor) and factor > 1
    ratio = [a / b for a, b in zip(freqs, O.plain_frequencies(rot["dims"], rot["base"]))]
    assert ratio[0] == 1.0 and any(0.21 < r < 0.99 for r in ratio)  # kept, and on the ramp
    plain = {"dims": 8, "base": 50.0}
    spec = RotarySpec.from_dict(plain, True)
    assert spec.frequencies() == pytest.approx(O.rotation(plain)[0]) and spec.amplitude == 1.0 and spec.to_dict() == plain


def test_no_training_path():
    with pytest.raises(NotImplementedError):
        CausalLM(preset("tiny-golonex"))
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-golonex"), dtype=torch.float32)(None)


def test_step_order_and_plan(monkeypatch):
    from verl_b200.models import hybrid

    model = build_model(ModelConfig.from_hf_dict(M.config([
        M.rglru(64, 2, 3), M.latent(2, 16, 16, 16, 32, 24, 40), M.latent(2, 16, 16, 16, 32, 24, 7)], width=64)), dtype=torch.float32)
    short = model.latent_short
    counts, ctx = [5, short + 1, 1, short, 300, 1, 200], [50, 90, 1, 700, 300, 80, 260]
    order = model.latent_order(counts)
    assert order == [2, 5, 0, 3, 1, 4, 6]  # single tokens, short portions, long ones
    monkeypatch.setattr(hybrid, "LATENT_GROUP", 400)
    plan = model.plan_latent([counts[i] for i in order], [ctx[i] for i in order], lambda v: v)
    assert (plan.short_seqs, plan.short_rows, plan.groups) == (4, 7 + short, ())
    # contexts: what a window reaches from the first new token, at most the sequence
    n1 = short + 1
    assert plan.groups_of(40) == ((4, 6, [0, n1 + 39, n1 + 339], n1 + 339, 300), (6, 7, [0, 239], 239, 200))
    assert plan.groups_of(7) == ((4, 6, [0, n1 + 6, n1 + 306], n1 + 306, 300), (6, 7, [0, 206], 206, 200))
    only = build_model(ModelConfig.from_hf_dict(M.CONFIGS["recurrent_only"]), dtype=torch.float32)
    assert only.latent_order([3, 1, 2]) == [1, 0, 2] and only.plan_latent([1], [1], None) is None
    att = build_model(ModelConfig.from_hf_dict(M.CONFIGS["attention_only"]), dtype=torch.float32)
    assert att.latent_order([3, 1, 2]) is None


# ------------------------------------------------------------------------------------------------------ operations on the CPU
@pytest.mark.parametrize("score,renormalize", [("sigmoid", False), ("softmax", False), ("softmax", True)])
def test_routing(score, renormalize):
    z, E, top = rand(9, 8, seed=1, scale=2.0), 6, 3
    counters = torch.zeros(E + 1, dtype=torch.int32)
    r = ops.moe_route(z, E, top, counters, score=score, renormalize=renormalize)
    s = torch.sigmoid(z[:, :E]) if score == "sigmoid" else torch.softmax(z[:, :E], -1)
    w, idx = s.topk(top, -1)
    assert torch.equal(r.idx, idx) and torch.allclose(r.weight, w / w.sum(-1, keepdim=True) if renormalize else w)
    assert len(set(r.dest.flatten().tolist())) == 9 * top
    for t in range(9):
        for k in range(top):
            assert int(r.blk_expert[int(r.dest[t, k]) // 128]) == int(idx[t, k])
    with pytest.raises(ValueError, match="score"):
        ops.moe_route(z, E, top, counters, score="tanh")


def test_linear_recurrent_unit_with_a_padding_row():
    """A row without a slot leaves every state alone."""
    W, taps = 12, 3
    proj, ring, state = rand(2, 2 * W, seed=1), rand(2, taps, W, seed=2), rand(2, W, seed=3)
    r0, s0 = ring.clone(), state.clone()
    out = ops.rglru(proj, rand(W, taps), rand(W), rand(4, 6, 6), rand(4, 6), rand(W), ring, state,
                    torch.tensor([0, 1, 2], dtype=torch.int32), torch.tensor([4, 1], dtype=torch.int32),
                    torch.tensor([1, -1], dtype=torch.int32), 1)
    assert torch.equal(ring[0], r0[0]) and torch.equal(state[0], s0[0]) and float(out[1].abs().sum()) == 0
    assert torch.equal(ring[1, 0], proj[0, W:]) and not torch.equal(state[1], s0[1])


# ------------------------------------------------------------------------------------------------------------------- engine
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_engine_portions_match_the_oracle(name, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg)
    eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"))
    ids = tokens(75, cfg["vocab"])
    want = O.forward(cfg, w, ids)
    for sizes in ([75], [1], [2], [40, 2, 33, 1]):  # the same engine: pages and slots a second time
        assert M.error(M.feed_portions(eng, "a", ids, sizes), want) < 1e-4, sizes
    assert eng.sched.stats()["free_pages"] == eng.num_blocks


def test_layers_one_by_one(tmp_path):
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=3, clear=False)
    eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"))
    ids = tokens(50, cfg["vocab"], 4)
    _, streams = O.forward(cfg, w, ids, keep_layers=True)
    seen = []
    eng.observe_layers = lambda i, x: seen.append(x)
    eng.feed([("a", ids, [])], ["a"])
    assert len(seen) == len(streams)
    assert all(float((a - b).abs().max() / b.std()) < 1e-4 for a, b in zip(seen, streams))


@pytest.mark.parametrize("short", [1, 2, 32])
def test_engine_mixed_steps_and_paused_requests(short, tmp_path):
    """Whatever form of latent attention a portion takes, and however its rows were reordered for it."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=2)
    eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"), num_blocks=16, max_model_len=256)
    eng.model.latent_short = short
    ids = {r: tokens(n, cfg["vocab"], k) for k, (r, n) in enumerate((("a", 60), ("b", 23), ("c", 90), ("d", 41), ("e", 64)))}
    want = {r: O.forward(cfg, w, t) for r, t in ids.items()}
    plan = [[("a", 40), ("b", 1)], [("b", 1), ("c", 33)], [("a", 1), ("b", 2), ("c", 1)], [("c", 30), ("d", 2)], [("b", 19)],
            [("a", 19), ("c", 26), ("d", 1)], [("d", 38), ("e", 64)]]
    at = dict.fromkeys(ids, 0)
    for step in plan:
        entries, rows, end = [], [], []
        for r, n in step:
            keep = list(range(n))[::-1] if r == "c" else list(range(0, n, 2))  # any places, in any order
            entries.append((r, ids[r][at[r]:at[r] + n], keep))
            rows.append(want[r][at[r]:at[r] + n][keep])
            at[r] += n
            if at[r] == len(ids[r]):
                end.append(r)
        assert M.error(eng.feed(entries, end), torch.cat(rows)) < 1e-4
    assert all(at[r] == len(ids[r]) for r in ids) and eng.sched.stats()["free_pages"] == eng.num_blocks


def greedy(cfg, w, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt):]


SMALL = M.config([M.rglru(48, 3, 3, M.moe(4, 2, 24, 32)), M.latent(2, 16, 8, 16, 24, 16, 13),
                  M.attention(2, 1, 16, 11, mlp=M.moe(3, 1, 32, 16))], vocab=64, width=48, side=8)


@pytest.mark.parametrize("kw", [{}, {"decode_burst": 1}, {"max_num_batched_tokens": 16}, {"num_blocks": 10}, {"max_num_seqs": 2}])
def test_greedy_generation(kw, tmp_path):
    """Through generate() and its scheduler: bursts, portions of prompts, preemption (10 pages where 16 are needed: states are
    rebuilt), waiting (slots change hands)."""
    w = M.weights(SMALL, seed=5)
    eng = M.engine(M.load_model(SMALL, w, tmp_path, torch.float32, "cpu"), max_model_len=96, **kw)
    prompts = [tokens(n, 64, n) for n in (21, 5, 33, 14)]
    n = 40 if "num_blocks" in kw else 12
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True))
    assert [o.token_ids for o in outs] == [greedy(SMALL, w, p, n) for p in prompts]
    if "num_blocks" in kw:
        assert sum(o.num_preempted for o in outs) > 0


def test_prefix_cache_only_without_recurrent_state(tmp_path):
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    p = tokens(70, 64)
    for cfg in (SMALL, M.config([M.latent(2, 16, 8, 16, 24, 16, 30), M.attention(2, 1, 16, 23, mlp=M.moe(3, 1, 32, 16))], vocab=64,
                                width=48, side=8)):
        w = M.weights(cfg, seed=5)
        eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"))
        first = eng.generate([p], sp)[0].token_ids
        outs = eng.generate([p, p[:50] + [1, 2, 3]], sp)
        assert outs[0].token_ids == first == greedy(cfg, w, p, 6) and outs[1].token_ids == greedy(cfg, w, p[:50] + [1, 2, 3], 6)
        assert (eng.sched.stats()["prefix_hits"] > 0) == (cfg is not SMALL)


def test_update_weights_and_command_line(tmp_path):
    from verl_b200.trainer import main_generation

    w0, w1 = M.weights(SMALL, seed=1), M.weights(SMALL, seed=2)
    eng = M.engine(M.load_model(SMALL, w0, tmp_path / "m0", torch.float32, "cpu"))
    eng.update_weights(w1.items())
    ids = tokens(30, 64)
    assert M.error(M.feed_portions(eng, "a", ids, [30]), O.forward(SMALL, w1, ids)) < 1e-4
    M.save(SMALL, w1, tmp_path / "m1")
    (tmp_path / "p.jsonl").write_text(json.dumps({"prompt": "1 2 3 4 5"}) + "\n")
    main_generation.main([f"model.path={tmp_path / 'm1'}", f"data.path={tmp_path / 'p.jsonl'}", "trainer.device=cpu",
                          f"data.output_path={tmp_path / 'o.jsonl'}", "rollout.response_length=5", "rollout.prompt_length=64",
                          "rollout.do_sample=false", "rollout.max_num_seqs=2"])
    assert len(json.loads((tmp_path / "o.jsonl").read_text())["responses"]) == 1


def test_preset_runs():
    eng = M.engine(build_model(preset("tiny-golonex"), dtype=torch.float32, seed=3))
    outs = eng.generate([[5, 6, 7], [8] * 50], SamplingParams(temperature=1.0, max_tokens=4, ignore_eos=True))
    assert [len(o.token_ids) for o in outs] == [4, 4] and all(np.isfinite(o.log_probs).all() for o in outs)
