"""Replay of a token trace through the serving engine: given tokens in, logits out, nothing sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Steps are JSON objects, one per line of standard input:

    {"step": 0, "entries": [{"id": "first", "tokens": [12, 7, 40, 9], "want": [1, 3]}], "end": []}

``entries`` names, per request, its next tokens and the places among them whose logits are wanted; ``end`` the requests
that are finished after the step. The entries of a step run as one batch on the engine's slots and cache pool
(``ServingEngine.attach`` / ``advance`` / ``detach``). Wanted logits go to ``OUT/<step>.f32``, little-endian fp32 in the
order of the entries; ``done <step>`` is printed after every step. The pool holds ``--max-tokens`` tokens, every
request's count rounded up to whole blocks; four requests may be live at a time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np
import torch

MAX_LIVE = 4


def build_engine(model, max_tokens: int):
    """Engine whose pool has room for ``max_tokens`` cached tokens in all."""
    from .engine import ServingEngine
    block = int(getattr(model.config, "block_size", 16) or 16)
    blocks = -(-int(max_tokens) // block)
    return ServingEngine(model, max_num_seqs=MAX_LIVE, max_model_len=blocks * block, num_blocks=blocks)


def run_step(engine, step: dict):
    """Advance the engine by one step; returns the wanted logits ``[n, vocab]`` (fp32, host) or None."""
    entries = step.get("entries") or []
    ids = [str(e["id"]) for e in entries]
    if len(set(ids)) != len(ids):
        raise ValueError(f"step {step.get('step')}: a request has two entries")
    for rid in ids:
        if rid not in engine._by_id:
            engine.attach(rid)
    got = engine.advance({r: e["tokens"] for r, e in zip(ids, entries)}, {r: e.get("want") or [] for r, e in zip(ids, entries)})
    rows = [got[r] for r in ids if got.get(r) is not None and len(got[r])]
    out = torch.cat(rows).float().cpu().numpy() if rows else None
    for rid in step.get("end") or []:
        engine.detach(str(rid))
    return out


def replay(engine, lines, out_dir: str, stdout=None):
    stdout = stdout or sys.stdout
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = run_step(engine, step)
        if logits is not None:
            np.ascontiguousarray(logits, dtype="<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        engine.model._check_device_status()
        stdout.write(f"done {step['step']}\n")
        stdout.flush()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace through the serving engine")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the cache pool, in tokens")
    a = ap.parse_args(argv)
    if not torch.cuda.is_available():
        raise RuntimeError("no CUDA device: the kernels are sm_100a code")
    from ..models.auto import AutoConfig, AutoModel, _classes_for
    from ..ops import _lib
    from ..ops import build as kernels
    config = AutoConfig.from_pretrained(a.model)
    _lib.use_library(kernels.ensure(_classes_for(config.to_dict())[1].kernel_sources))
    model = AutoModel.from_pretrained(a.model, config=config, dtype=a.dtype, strict=True).eval()
    replay(build_engine(model, a.max_tokens), iter(sys.stdin.readline, ""), a.out)
    return 0


if __name__ == "__main__":
    sys.exit(main())
