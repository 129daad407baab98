"""The Padodra design in the framework, without a GPU: configuration and registry, checkpoints, the plan of latent attention,
the engine's batching, and greedy generation, against the plain implementation in ``_padodra_oracle.py``."""

import json
import math

import numpy as np
import pytest
import torch

import _padodra_models as M
import _padodra_oracle as O
from verl_b200 import ops
from verl_b200.models import CausalLM, ModelConfig, build_model, preset
from verl_b200.models.hf_io import load_hf_checkpoint, native_to_hf_state_dict, save_hf_checkpoint
from verl_b200.models.layer_specs import RotarySpec
from verl_b200.rollout import SamplingParams


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@pytest.mark.parametrize("dims,base,scaling", [
    (64, 3000.0, M.LLAMA3), (16, 5e5, {"factor": 8.0, "high": 4.0, "low": 1.0, "original": 8192}),
    (32, 100.0, {"factor": 3.0, "high": 1.25, "low": 1.0, "original": 64}), (2, 10.0, M.LLAMA3)])
def test_llama3_frequencies(dims, base, scaling):
    spec = RotarySpec.from_dict({"dims": dims, "base": base, "scaling": scaling}, True)
    assert spec.frequencies() == pytest.approx(O.llama3_frequencies(dims, base, scaling), rel=1e-12) and spec.amplitude == 1.0
    assert spec.interleaved and spec.to_dict() == {"dims": dims, "base": base, "scaling": scaling}


def test_llama3_bands():
    """The three bands are all there: kept, blended, slowed down."""
    f = O.plain_frequencies(64, 3000.0)
    g = RotarySpec.from_dict({"dims": 64, "base": 3000.0, "scaling": M.LLAMA3}, True).frequencies()
    ratio = [a / b for a, b in zip(g, f)]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 6) and any(1 / 6 + 1e-3 < r < 1 - 1e-3 for r in ratio)


@pytest.mark.parametrize("dims,base,scaling", [
    (64, 2000.0, M.YARN), (16, 5e5, {"factor": 40.0, "fast": 32.0, "original": 4096, "slow": 1.0}),
    (8, 50.0, {"factor": 4.0, "fast": 2.0, "original": 32, "slow": 2.0}),    # a ramp of (almost) no width
    (8, 1e4, {"factor": 4.0, "fast": 900.0, "original": 64, "slow": 0.01})])  # both ends outside: clamped
def test_yarn_frequencies(dims, base, scaling):
    spec = RotarySpec.from_dict({"dims": dims, "base": base, "scaling": scaling}, False)
    freqs, factor = O.yarn_frequencies(dims, base, scaling)
    assert spec.frequencies() == pytest.approx(freqs, rel=1e-12) and spec.amplitude == pytest.approx(factor)
    assert factor == pytest.approx(0.1 * math.log(scaling["factor"]) + 1)


def test_bad_rotations_are_refused():
    with pytest.raises(ValueError, match="even"):
        RotarySpec.from_dict({"dims": 7, "base": 10.0}, True)
    with pytest.raises(ValueError, match="scaling"):
        RotarySpec.from_dict({"dims": 8, "base": 10.0, "scaling": {"factor": 2.0, "original": 8}}, True)


@pytest.mark.parametrize("interleaved", [True, False])
def test_rotation_keeps_lengths_and_relative_angles(interleaved):
    freqs = O.llama3_frequencies(12, 100.0, M.LLAMA3)
    x = torch.randn(1, 1, 20, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    y = O.rotate(x.expand(40, 1, 20), freqs, interleaved)
    assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1)) and torch.equal(y[:, 0, 12:], x.expand(40, 1, 20)[:, 0, 12:])
    dots = torch.einsum("id,jd->ij", y[:, 0], y[:, 0])
    assert torch.allclose(dots[5, 9], dots[30, 34]) and not torch.allclose(dots[5, 9], dots[5, 10])
    got = ops.attention.rotate_pairs(x.float().expand(40, 1, 20), torch.arange(40), torch.tensor(freqs), interleaved)
    assert torch.allclose(got, y.float(), atol=1e-5)


def test_oracle_softmax_sink_and_cap():
    s = torch.tensor([[0.3, -1.0, 2.0]], dtype=torch.float64)
    assert torch.allclose(O.softmax_with_sink(s), torch.softmax(s, -1))
    w = O.softmax_with_sink(s, 1.5)
    assert torch.allclose(w, torch.softmax(torch.cat([s, torch.tensor([[1.5]], dtype=torch.float64)], -1), -1)[:, :3])
    assert float(O.softcap(torch.tensor(1e6), 7.0)) == pytest.approx(7.0)


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_config_and_checkpoint_round_trip(name, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg)
    mc, native = load_hf_checkpoint(M.save(cfg, w, tmp_path / "a"))
    assert mc.model_type == "padodra" and mc.is_layer_list and not mc.has_recurrent_state and mc.to_hf_dict() == cfg
    assert mc.num_parameters() == sum(t.numel() for t in w.values())
    back = native_to_hf_state_dict(mc, native)
    assert back.keys() == w.keys() and all(torch.equal(back[k], w[k]) for k in w)
    save_hf_checkpoint(mc, native, tmp_path / "b")
    mc2, native2 = load_hf_checkpoint(tmp_path / "b")
    assert mc2 == mc and all(torch.equal(native2[k], native[k]) for k in native)


def test_bad_configurations_are_refused(tmp_path):
    def changed(layer, key, value, part="mixer"):
        cfg = json.loads(json.dumps(M.CONFIGS["mixed"]))
        cfg["layers"][layer][part][key] = value
        return cfg

    for cfg, why in ((changed(1, "kv_heads", 4), "multiple"), (changed(0, "rot_dim", 8), "rotated"),
                     (changed(1, "rot", {"dims": 64, "base": 10.0}), "rotated"), (changed(1, "kind", "sparse", "mlp"), "kind")):
        with pytest.raises(ValueError, match=why):
            ModelConfig.from_hf_dict(cfg)
    with pytest.raises(ValueError, match="rows"):
        load_hf_checkpoint(M.save(changed(0, "kv_rank", 40), M.weights(M.CONFIGS["mixed"]), tmp_path))


def test_no_training_path():
    with pytest.raises(NotImplementedError):
        CausalLM(preset("tiny-padodra"))
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-padodra"), dtype=torch.float32)(None)


def test_latent_plan(monkeypatch):
    from verl_b200.models import hybrid

    model = build_model(preset("tiny-padodra"), dtype=torch.float32)
    short = model.latent_short
    counts, ctx = [5, short + 1, 1, short, 300, 200], [50, 90, 1, 700, 300, 260]
    order = model.latent_order(counts)
    assert order == [0, 2, 3, 1, 4, 5]
    monkeypatch.setattr(hybrid, "LATENT_GROUP", 400)
    plan = model.plan_latent([counts[i] for i in order], [ctx[i] for i in order], lambda v: v)
    assert (plan.short_seqs, plan.short_rows) == (3, 6 + short)
    assert plan.groups == ((3, 5, [0, 90, 390], 390, 300), (5, 6, [0, 260], 260, 200))
    plain = build_model(preset("tiny-fuganex"), dtype=torch.float32)
    assert plain.latent_order(counts) is None and plain.plan_latent(counts, ctx, None) is None


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_engine_portions_match_the_oracle(name, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg)
    eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"))
    ids = tokens(75, cfg["vocab"])
    want = O.forward(cfg, w, ids)
    for sizes in ([75], [1], [2], [40, 2, 33, 1]):  # the same engine: pages are used again
        assert M.error(M.feed_portions(eng, "a", ids, sizes), want) < 1e-4, sizes
    assert eng.sched.stats()["free_pages"] == eng.num_blocks


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


SMALL = M.config([M.attention(2, 1, 16, 16, 11, ff=48), M.latent(2, 16, 8, 16, 24)], vocab=64, width=48)


@pytest.mark.parametrize("kw", [{}, {"decode_burst": 1}, {"max_num_batched_tokens": 16},
                                {"num_blocks": 10, "enable_prefix_caching": False}, {"max_num_seqs": 2}])
def test_greedy_generation(kw, tmp_path):
    """Through generate() and its scheduler: bursts, portions of prompts, preemption (10 pages where 16 are needed), waiting."""
    w = M.weights(SMALL, seed=5)
    eng = M.engine(M.load_model(SMALL, w, tmp_path, torch.float32, "cpu"), max_model_len=96, **kw)
    prompts = [tokens(n, 64, n) for n in (21, 5, 33, 14)]
    n = 40 if "num_blocks" in kw else 12
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True))
    assert [o.token_ids for o in outs] == [greedy(SMALL, w, p, n) for p in prompts]
    if "num_blocks" in kw:
        assert sum(o.num_preempted for o in outs) > 0


def test_prefix_cache(tmp_path):
    """Chunks are counted from the sequence's start and latents carry their position: pages can be shared."""
    w = M.weights(SMALL, seed=5)
    eng = M.engine(M.load_model(SMALL, w, tmp_path, torch.float32, "cpu"))
    p = tokens(70, 64)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    first = eng.generate([p], sp)[0].token_ids
    outs = eng.generate([p, p[:50] + [1, 2, 3]], sp)
    assert outs[0].token_ids == first == greedy(SMALL, w, p, 6) and outs[1].token_ids == greedy(SMALL, w, p[:50] + [1, 2, 3], 6)
    assert eng.sched.stats()["prefix_hits"] > 0


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
    eng = M.engine(build_model(preset("tiny-padodra"), dtype=torch.float32, seed=3))
    outs = eng.generate([[5, 6, 7], [8] * 50], SamplingParams(temperature=1.0, max_tokens=4, ignore_eos=True))
    assert [len(o.token_ids) for o in outs] == [4, 4] and all(np.isfinite(o.log_probs).all() for o in outs)
