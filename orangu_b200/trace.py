"""Replays a trace: token ids of several requests, step by step, through a model's slot pool; logits of the places asked for.

One JSON object a line on standard input:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
All entries of a step are one batch.  A request takes a slot at its first entry and gives it, its pages and its state back after
the step that lists it under "end".  Logits go to <out>/<step>.f32, and "done <step>" to standard output when the step has run."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

SLOTS = 4               # requests alive at a time
REQUEST_ROUNDING = 64   # every live request counts as a multiple of this many tokens
MAX_STEP_ROWS = 8192    # longer steps run in portions


def run_step(pool, held: dict, step: dict):
    """One step through the pool; the wanted logits in the order of the entries and of their places."""
    guards, lists, flat, at = [], [], [], 0
    for e in step["entries"]:
        if e["id"] not in held:
            guard = pool.try_acquire(0)
            if guard is None:
                raise RuntimeError(f"request {e['id']}: no free slot")
            held[e["id"]] = guard
        guards.append(held[e["id"]])
        lists.append(e["tokens"])
        flat += [at + w for w in e.get("want", [])]
        at += len(e["tokens"])
    if not guards:
        return None
    rows = sorted(set(flat))
    logits = pool.forward(guards, lists, rows)
    return logits[np.searchsorted(rows, flat)] if flat else None


def replay(model, lines, out_dir: str, max_tokens: int, emit) -> None:
    from .scheduler import SlotPool

    pool = SlotPool(model, SLOTS, max_tokens)
    held = {}
    try:
        for line in lines:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = run_step(pool, held, step)
            for name in step.get("end", []):
                if name in held:
                    held.pop(name).release()
            if logits is not None:
                np.ascontiguousarray(logits, "<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
            emit(f"done {step['step']}")
    finally:
        pool.close()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a .gguf file")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    a = ap.parse_args(argv)

    from . import CudaBackend, build
    from .registry import load_model

    build.ensure_for(a.model)
    tokens = -(-a.max_tokens // REQUEST_ROUNDING) * REQUEST_ROUNDING
    model = load_model(CudaBackend.init(0), a.model, dtype=a.dtype, max_seq_len=tokens, max_batch_tokens=min(tokens, MAX_STEP_ROWS),
                       kv_pool_tokens=tokens, state_slots=SLOTS)

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(model, iter(sys.stdin.readline, ""), a.out, tokens, emit)
    model.close()
    return 0
