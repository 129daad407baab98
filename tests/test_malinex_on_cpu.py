"""The Malinex design in the framework, without a GPU: configuration and registry, checkpoints, shared weights, the engine's
batching and states, and greedy generation, against the plain implementation in ``_malinex_oracle.py``."""

import json
import math

import numpy as np
import pytest
import torch

import _malinex_models as M
import _malinex_oracle as O
from verl_b200 import ops
from verl_b200.models import CausalLM, ModelConfig, build_model, preset
from verl_b200.models.hf_io import load_hf_checkpoint, native_to_hf_state_dict, save_hf_checkpoint
from verl_b200.models.registry import ModelRegistry
from verl_b200.rollout import SamplingParams


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


# ------------------------------------------------------------------------------------------- the oracle against other forms
def test_oracle_linear_attention():
    """The recurrence against its unrolled sum, and continued from a state."""
    T, H, D, V = 9, 2, 4, 3
    q, k, v, z = rand(T, H, D, seed=1), rand(T, H, D, seed=2), rand(T, H, V, seed=3), rand(T, H, D, seed=4, scale=3.0)
    a = O.decays(z, 2.5)
    assert torch.allclose(a, torch.sigmoid(z) ** (1 / 2.5))
    o, S = O.linear_attention(q, k, v, a)
    for t in (0, 1, 5, 8):
        want = torch.zeros(H, V)
        for s in range(t + 1):
            gone = a[s + 1:t + 1].prod(0) if s < t else torch.ones(H, D)
            want += (q[t] * k[s] * gone).sum(-1)[:, None] * v[s]
        assert torch.allclose(o[t], want, atol=1e-5)
    o1, S1 = O.linear_attention(q[:4], k[:4], v[:4], a[:4])
    o2, S2 = O.linear_attention(q[4:], k[4:], v[4:], a[4:], S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)
    assert torch.isfinite(O.decays(torch.tensor([-1e4, 1e4, -80.0]), 1.0)).all()


def test_oracle_sigmoid_attention():
    T, H, D = 5, 2, 4
    q, k, v = rand(T, H, D, seed=1), rand(T, 1, D, seed=2), rand(T, 1, 3, seed=3)
    r1, r2, shift = torch.tensor([0.0, 1.5]), torch.tensor([0.3, 0.4]), torch.tensor([-1.0, 0.5])
    out = O.sigmoid_attend(q, k, v, 0.5, O.distance_bias(T, r1, r2), shift)
    for i in range(T):
        for h in range(H):
            want = sum(torch.sigmoid(q[i, h] @ k[j, 0] * 0.5 - r1[h] * math.log(1 + r2[h] * (i - j)) + shift[h]) * v[j, 0]
                       for j in range(i + 1))
            assert torch.allclose(out[i, h], want, atol=1e-6)


def test_oracle_temperature_and_routing():
    t = O.query_temperature([0, 28, 29, 58, 59, 89], {"coef": 0.5, "every": 30})
    want = [1, 1, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(4)]
    assert t.tolist() == pytest.approx(want)
    assert O.query_temperature([0, 1], {"coef": 1.0, "every": 1}).tolist() == pytest.approx([1 + math.log(2), 1 + math.log(3)])
    idx, w = O.route(torch.zeros(1, 3), torch.zeros(4, 3), torch.tensor([0.0, 0.3, 0.1, 0.2]), 2)
    assert idx.tolist() == [[1, 3]] and torch.allclose(w, torch.full((1, 2), 0.5))
    x = rand(50, seed=1, scale=2.0)
    assert torch.allclose(O.gelu(x), torch.nn.functional.gelu(x), atol=1e-6) and torch.equal(O.relu2(x), torch.relu(x) ** 2)


# ------------------------------------------------------------------------------------- configuration, registry, checkpoints
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_config_and_checkpoint_round_trip(name, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg)
    mc, native = load_hf_checkpoint(M.save(cfg, w, tmp_path / "a"))
    assert mc.model_type == "malinex" and mc.is_layer_list and not mc.tie_word_embeddings and mc.to_hf_dict() == cfg
    assert mc.has_recurrent_state == any(x["type"] == "gla" for x in cfg["layers"])
    assert mc.max_position_embeddings == cfg["max_positions"]
    assert mc.num_parameters() == sum(t.numel() for t in w.values())
    back = native_to_hf_state_dict(mc, native)
    assert back.keys() == w.keys() and all(torch.equal(back[k], w[k]) for k in w)
    save_hf_checkpoint(mc, native, tmp_path / "b")
    mc2, native2 = load_hf_checkpoint(tmp_path / "b")
    assert mc2 == mc and all(torch.equal(native2[k], native[k]) for k in native)


def test_sizes_that_the_tensors_give(tmp_path):
    cfg = json.loads(json.dumps(M.CONFIGS["mixed"]))
    w = M.weights(cfg)
    del cfg["max_positions"]
    mc, _ = load_hf_checkpoint(M.save(cfg, w, tmp_path))
    assert mc.max_position_embeddings == 600
    ranks = [s.mixer.rank for s in mc.layer_specs if s.kind == "gla"]
    assert ranks == [M.RANKS[0], M.RANKS[0], M.RANKS[3], M.RANKS[3]]  # two of them the layers of others


def test_registry():
    assert ModelRegistry.family("Malinex") == "malinex"
    build = ModelRegistry.load_model_cls("Malinex")
    assert type(build(preset("tiny-malinex"), dtype=torch.float32)).__name__ == "HybridLM"


def test_bad_configurations_are_refused(tmp_path):
    def changed(layer, key, value, part=None):
        cfg = json.loads(json.dumps(M.CONFIGS["mixed"]))
        at = cfg["layers"][layer]
        (at if part is None else at[part])[key] = value
        return cfg

    for cfg, why in ((changed(1, "kv_heads", 4, "mixer"), "multiple"), (changed(0, "kind", "sparse", "mlp"), "kind"),
                     (changed(1, "router", {"experts": 3, "top": 4}, "mlp"), "experts"), (changed(0, "type", "lstm"), "layer type"),
                     (changed(1, "q_temp", {"coef": 1.0, "every": 0}, "mixer"), "temperature"),
                     (changed(2, "weights_of", 9), "weights of"), (changed(2, "weights_of", 1), "weights of"),
                     (changed(0, "weights_of", 2), "weights of")):
        with pytest.raises(ValueError, match=why):
            ModelConfig.from_hf_dict(cfg)
    for cfg in (changed(1, "vdim", 16, "mixer"), changed(0, "ff", 152, "mlp"), changed(3, "vdim", 24, "mixer")):
        with pytest.raises(ValueError, match="rows"):
            load_hf_checkpoint(M.save(cfg, M.weights(M.CONFIGS["mixed"]), tmp_path))


def test_layers_share_weights(tmp_path):
    """A layer with another's weights has no parameters of its own, in memory and in the state dict, but a cache of its own."""
    cfg = M.CONFIGS["mixed"]
    model = M.load_model(cfg, M.weights(cfg), tmp_path, torch.float32, "cpu")
    assert model.runs[2] is model.runs[0] and model.runs[4] is model.runs[1] and model.runs[5] is model.runs[3]
    assert [x is None for x in model.layers] == [False, False, True, False, True, True, False]
    assert not any(n.startswith(("layers.2.", "layers.4.", "layers.5.")) for n in model.state_dict())
    assert sum(p.numel() for p in model.parameters()) >= model.cfg.num_parameters()  # rows that fill up to a multiple of eight
    eng = M.engine(model)
    layers = eng.state_cache.layers
    assert len(layers) == 7 and layers[0][0].data_ptr() != layers[2][0].data_ptr() and layers[1][0].data_ptr() != layers[4][0].data_ptr()


def test_no_training_path():
    with pytest.raises(NotImplementedError):
        CausalLM(preset("tiny-malinex"))
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-malinex"), dtype=torch.float32)(None)


def test_step_order():
    model = build_model(ModelConfig.from_hf_dict(M.config([M.attention(2, 1, 16, 16), M.gla(2, 16, 16)], width=64)), dtype=torch.float32)
    assert model.latent_order([5, 1, 30, 1, 2]) == [1, 3, 0, 2, 4]  # single tokens first
    att = build_model(ModelConfig.from_hf_dict(M.CONFIGS["attention_only"]), dtype=torch.float32)
    assert att.latent_order([3, 1, 2]) is None


# ------------------------------------------------------------------------------------------------------ operations on the CPU
def test_corrected_routing():
    z, E, top = rand(9, 8, seed=1, scale=2.0), 6, 3
    corr = torch.tensor([0.5, 0.0, -0.4, 0.2, 0.0, 0.1])
    r = ops.moe_route(z, E, top, torch.zeros(E + 1, dtype=torch.int32), score="softmax", renormalize=True, correction=corr)
    s = torch.softmax(z[:, :E], -1)
    idx = (s + corr).topk(top, -1).indices
    w = s.gather(1, idx)
    assert torch.equal(r.idx, idx) and torch.allclose(r.weight, w / w.sum(-1, keepdim=True))


def test_linear_attention_with_a_padding_row():
    """A row without a slot leaves every state alone."""
    H, D, V, R = 2, 4, 6, 3
    proj, state = rand(2, 2 * H * (D + V) + R, seed=1), rand(2, H, V, D, seed=2)
    s0 = state.clone()
    out = ops.gated_linear_attention(proj, rand(H * D, R), rand(H * D), rand(V), state, torch.tensor([0, 1, 2], dtype=torch.int32),
                                     torch.tensor([4, 1], dtype=torch.int32), torch.tensor([1, -1], dtype=torch.int32), 1, H, D, V,
                                     4.0, 1e-6)
    assert torch.equal(state[0], s0[0]) and float(out[1].abs().sum()) == 0 and not torch.equal(state[1], s0[1])


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


def test_engine_mixed_steps_and_paused_requests(tmp_path):
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, seed=2)
    eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"), num_blocks=16, max_model_len=256)
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


SMALL = M.config([M.gla(2, 16, 24, 3.0, M.moe(4, 2, 24, 32)), M.attention(2, 1, 16, 16, (0.5, 9), mlp=M.dense(40)), 0], vocab=64, width=48,
                 positions=90)


@pytest.mark.parametrize("kw", [{}, {"decode_burst": 1}, {"max_num_batched_tokens": 16}, {"num_blocks": 10}, {"max_num_seqs": 2}])
def test_greedy_generation(kw, tmp_path):
    """Through generate() and its scheduler: bursts, portions of prompts, preemption (10 pages where 16 are needed: states are
    rebuilt), waiting (slots change hands)."""
    w = M.weights(SMALL, seed=5)
    eng = M.engine(M.load_model(SMALL, w, tmp_path, torch.float32, "cpu"), **kw)
    prompts = [tokens(n, 64, n) for n in (21, 5, 33, 14)]
    n = 40 if "num_blocks" in kw else 12
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True))
    assert [o.token_ids for o in outs] == [greedy(SMALL, w, p, n) for p in prompts]
    if "num_blocks" in kw:
        assert sum(o.num_preempted for o in outs) > 0


def test_no_sequence_outgrows_the_position_table(tmp_path):
    w = M.weights(SMALL, seed=5)
    eng = M.engine(M.load_model(SMALL, w, tmp_path, torch.float32, "cpu"))
    assert eng.max_model_len == 90
    out = eng.generate([tokens(80, 64)], SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))[0]
    assert out.token_ids == greedy(SMALL, w, tokens(80, 64), len(out.token_ids)) and len(out.token_ids) == 10
    with pytest.raises(ValueError, match="does not fit"):
        eng.generate([tokens(91, 64)], SamplingParams(max_tokens=1))
    ids = tokens(90, 64, 7)
    assert M.error(M.feed_portions(eng, "a", ids, [60, 29, 1], end=False), O.forward(SMALL, w, ids)) < 1e-4
    with pytest.raises(Exception, match="max_model_len"):
        eng.feed([("a", [1], [0])])


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
    eng = M.engine(build_model(preset("tiny-malinex"), dtype=torch.float32, seed=3))
    outs = eng.generate([[5, 6, 7], [8] * 50], SamplingParams(temperature=1.0, max_tokens=4, ignore_eos=True))
    assert [len(o.token_ids) for o in outs] == [4, 4] and all(np.isfinite(o.log_probs).all() for o in outs)
