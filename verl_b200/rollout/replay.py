"""Replay a trace: feed given token ids through a model step by step and write the logits that the trace asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is one step: ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}``.
All entries of a step run as one batch of the rollout engine (:meth:`NativeRolloutEngine.feed`): portions of prompts next
to single tokens, from the pages and states that earlier steps left; ``end`` gives a request's pages and state back. The
logits at the ``want`` places go to ``OUT/<step>.f32`` ([wanted, vocab] little-endian fp32), then ``done <step>`` is
printed. Nothing is sampled.
"""

from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


def build_engine(model_dir: str, dtype_name: str, max_tokens: int, max_requests: int = 4, page_group: int = 64):
    """Engine with cache pages for ``max_tokens`` live tokens (a multiple of ``page_group`` tokens) and ``max_requests``
    state slots."""
    import torch

    from ..models import build_model
    from ..workers.engine_workers import resolve_model_config
    from .engine import NativeRolloutEngine

    if not torch.cuda.is_available():
        raise RuntimeError("a replay runs on the GPU kernels: no CUDA device is visible")
    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype_name]
    cfg, state = resolve_model_config({"path": model_dir})
    if state is None:
        raise FileNotFoundError(f"no safetensors file under {model_dir}")
    model = build_model(cfg, dtype=dtype, device="cuda", init=False)
    model.load_state_dict(state, strict=True)
    tokens = (max_tokens + page_group - 1) // page_group * page_group
    block = 16
    return NativeRolloutEngine(model, max_num_seqs=max_requests, max_model_len=tokens, max_num_batched_tokens=tokens,
                               block_size=block, num_blocks=tokens // block)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    from .. import _build

    _build.build()  # compiles what has changed since the last call
    import numpy as np

    from ..ops import _lib

    eng = build_engine(a.model, a.dtype, a.max_tokens)
    out = Path(a.out)
    out.mkdir(parents=True, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = eng.feed([(e["id"], e["tokens"], e["want"]) for e in step["entries"] if e["tokens"]],
                          step.get("end") or [])
        if logits is not None:
            logits.cpu().numpy().astype(np.dtype("<f4"), copy=False).tofile(out / f"{step['step']}.f32")
        code, blk, detail = _lib.read_status(eng.device)
        if code:
            raise RuntimeError(f"a kernel gave up waiting: code {code} (block {blk}, detail {detail})")
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
