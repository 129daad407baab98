"""The Fuganex design in the framework, without a GPU: configuration and registry, checkpoints, scheduler and state slots,
the engine's batching, and greedy generation, against the plain implementation in ``_fuganex_oracle.py``."""

import json

import numpy as np
import pytest
import torch

import _fuganex_models as M
import _fuganex_oracle as O
from verl_b200.models import ModelConfig, build_model, preset
from verl_b200.models.hf_io import hf_to_native_state_dict, load_hf_checkpoint, native_to_hf_state_dict, save_hf_checkpoint
from verl_b200.models.layer_specs import distance_buckets
from verl_b200.rollout import SamplingParams, Scheduler


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@pytest.mark.parametrize("rows,far", [(12, 40), (16, 128), (24, 96), (32, 512), (5, 33), (2, 7), (7, 20.5), (3, 2), (64, 4096)])
def test_distance_buckets(rows, far):
    got = distance_buckets(rows, far)
    assert got == [O.distance_bucket(n, rows, far) for n in range(len(got))]
    assert got[-1] == rows - 1 and O.distance_bucket(len(got) + 1000, rows, far) == rows - 1
    assert got == sorted(got)


def test_distance_buckets_on_exact_edges():
    # far / h = 8, m = 12: distances 2 h and 4 h lie exactly on the edges of rows h + 4 and h + 8
    got = distance_buckets(24, 96)
    assert [got[24], got[23], got[48], got[47]] == [16, 15, 20, 19]
    with pytest.raises(ValueError):
        distance_buckets(16, 8)


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_config_and_checkpoint_round_trip(name, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg)
    mc, native = load_hf_checkpoint(M.save(cfg, w, tmp_path / "a"))
    assert mc.model_type == "fuganex" and mc.is_layer_list and mc.to_hf_dict() == cfg
    assert mc.num_parameters() == sum(t.numel() for t in w.values())
    back = native_to_hf_state_dict(mc, native)
    assert back.keys() == w.keys() and all(torch.equal(back[k], w[k]) for k in w)
    save_hf_checkpoint(mc, native, tmp_path / "b")
    mc2, native2 = load_hf_checkpoint(tmp_path / "b")
    assert mc2 == mc and all(torch.equal(native2[k], native[k]) for k in native)


def test_bad_configurations_are_refused(tmp_path):
    cfg = json.loads(json.dumps(M.CONFIGS["mixed"]))
    cfg["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="layer type"):
        ModelConfig.from_hf_dict(cfg)
    cfg = json.loads(json.dumps(M.CONFIGS["mixed"]))
    w = M.weights(cfg)
    cfg["layers"][1]["mixer"]["heads"] = 4
    with pytest.raises(ValueError, match="rows"):
        load_hf_checkpoint(M.save(cfg, w, tmp_path))


def test_no_training_path():
    from verl_b200.models import CausalLM

    with pytest.raises(NotImplementedError):
        CausalLM(preset("tiny-fuganex"))
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-fuganex"), dtype=torch.float32)(None)


def test_scheduler_feed_and_state_slots():
    s = Scheduler(8, 16, 2, 64, 100, prefix_caching=False)
    assert s.feed([7, 9], [[1] * 20, [2]]) == (2, 21)
    a = s.step_state_slots(2).tolist()
    assert sorted(a) == [0, 1] and s.seq_start[:2].tolist() == [0, 0] and s.seq_prefill[:2].all()
    s.commit(np.full(2, -1, np.int64), np.zeros(2, np.int32))
    assert s.feed([9], [[3]]) == (1, 1) and s.seq_start[0] == 1 and not s.seq_prefill[0]
    assert s.step_state_slots(1)[0] == a[1]
    s.commit(np.full(1, -1, np.int64), np.zeros(1, np.int32))
    free = s.stats()["free_pages"]
    for sids, chunks, why in (([11], [[1]], "max_num_seqs"), ([7, 7], [[1], [1]], "twice"), ([7], [[1] * 70], "more tokens"),
                              ([7], [[]], "empty")):
        with pytest.raises(ValueError, match=why):
            s.feed(sids, chunks)
    assert s.stats()["free_pages"] == free  # a refused step changes nothing
    s.remove(7)
    assert s.stats()["free_pages"] == free + 2
    assert s.feed([11], [[1] * 60]) == (1, 60) and s.step_state_slots(1)[0] == a[0]  # the freed slot again


def test_scheduler_out_of_pages_is_refused():
    s = Scheduler(2, 16, 2, 64, 100, prefix_caching=False)
    with pytest.raises(ValueError, match="pages"):
        s.feed([1], [[1] * 33])
    assert s.feed([1], [[1] * 32]) == (1, 32)


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_engine_portions_match_the_oracle(name, tmp_path):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg)
    eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"))
    ids = tokens(75, cfg["vocab"])
    want = O.forward(cfg, w, ids)
    for sizes in ([75], [1], [2], [30, 2, 17, 1]):  # the same engine: pages and slots are used again
        assert M.error(M.feed_portions(eng, "a", ids, sizes), want) < 1e-4, sizes
    assert eng.sched.stats()["free_pages"] == eng.num_blocks


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
            entries.append((r, ids[r][at[r]:at[r] + n], list(range(n))))
            rows.append(want[r][at[r]:at[r] + n])
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


@pytest.mark.parametrize("kw", [{}, {"decode_burst": 1}, {"max_num_batched_tokens": 16}, {"num_blocks": 10}, {"max_num_seqs": 2}])
def test_greedy_generation(kw, tmp_path):
    """Through generate() and its scheduler: bursts, portions of prompts, preemption (10 pages where 16 are needed), waiting."""
    cfg = M.config([M.delta(2, 1, 16, 16, 3), M.attention(2, 1, 16, 16, 9, 2, bias_max=20, ff=48)], vocab=64, width=48)
    w = M.weights(cfg, seed=5)
    eng = M.engine(M.load_model(cfg, w, tmp_path, torch.float32, "cpu"), max_model_len=96, **kw)
    prompts = [tokens(n, 64, n) for n in (21, 5, 33, 14)]
    n = 40 if "num_blocks" in kw else 12
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True))
    assert [o.token_ids for o in outs] == [greedy(cfg, w, p, n) for p in prompts]
    if "num_blocks" in kw:
        assert sum(o.num_preempted for o in outs) > 0


def test_shared_prompts_are_not_taken_from_a_prefix_cache(tmp_path):
    """Recurrent state is not in the pages: two equal prompts must both run, whatever the caller asked for."""
    cfg = M.config([M.delta(2, 1, 16, 16, 3), M.attention(2, 1, 16, 16, 9, 2, bias_max=20)], vocab=64, width=48)
    eng = M.engine(M.load_model(cfg, M.weights(cfg), tmp_path, torch.float32, "cpu"), enable_prefix_caching=True)
    p = tokens(40, 64)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    a = eng.generate([p], sp)[0].token_ids
    assert eng.generate([p], sp)[0].token_ids == a and not eng.enable_prefix_caching


def test_update_weights_and_command_line(tmp_path):
    from verl_b200.trainer import main_generation

    cfg = M.config([M.attention(2, 1, 16, 16, 9, 2, bias_max=20, ff=48), M.delta(2, 1, 16, 16, 3)], vocab=64, width=48)
    w0, w1 = M.weights(cfg, seed=1), M.weights(cfg, seed=2)
    eng = M.engine(M.load_model(cfg, w0, tmp_path / "m0", torch.float32, "cpu"))
    eng.update_weights(w1.items())  # the derived bias tables follow
    ids = tokens(30, 64)
    assert M.error(M.feed_portions(eng, "a", ids, [30]), O.forward(cfg, w1, ids)) < 1e-4
    M.save(cfg, w1, tmp_path / "m1")
    (tmp_path / "p.jsonl").write_text(json.dumps({"prompt": "1 2 3 4 5"}) + "\n")
    main_generation.main([f"model.path={tmp_path / 'm1'}", f"data.path={tmp_path / 'p.jsonl'}", "trainer.device=cpu",
                          f"data.output_path={tmp_path / 'o.jsonl'}", "rollout.response_length=5", "rollout.prompt_length=64",
                          "rollout.do_sample=false", "rollout.max_num_seqs=2"])
    assert len(json.loads((tmp_path / "o.jsonl").read_text())["responses"]) == 1


def test_preset_runs():
    cfg = preset("tiny-fuganex")
    eng = M.engine(build_model(cfg, dtype=torch.float32, seed=3))
    outs = eng.generate([[5, 6, 7], [8] * 50], SamplingParams(temperature=1.0, max_tokens=4, ignore_eos=True))
    assert [len(o.token_ids) for o in outs] == [4, 4]
    assert native_to_hf_state_dict(cfg, hf_to_native_state_dict(cfg, native_to_hf_state_dict(cfg, dict(
        eng.model.state_dict())))).keys() == native_to_hf_state_dict(cfg, dict(eng.model.state_dict())).keys()
