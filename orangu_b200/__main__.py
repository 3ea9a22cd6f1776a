"""Command line.

    python -m orangu_b200 generate --model PATH --tokens 1,2,3 [--tokens 4,5] --n 32    greedy continuations, all prompts at once
    python -m orangu_b200 trace --model PATH --out DIR --max-tokens N                   replay a trace (see trace.py)
    python -m orangu_b200 build                                                          compile the native libraries
"""
from __future__ import annotations

import argparse
import sys
import threading


def generate(model, prompts, n: int, repeat_penalty: float = 1.0, repeat_last_n: int = 64, prefill_batch: int = 0):
    """Greedy continuations of several prompts, one thread per prompt through the slot pool as a server runs them."""
    from .scheduler import SlotPool

    longest = max(len(p) for p in prompts) + n
    pool = SlotPool(model, len(prompts), longest, prefill_batch=prefill_batch)
    out, errors = [None] * len(prompts), []

    def one(i):
        try:
            with pool.try_acquire() as slot:
                history = list(prompts[i])
                logits_penalised = repeat_penalty != 1.0
                if logits_penalised and len(history) > 1:  # the last prompt token is a decode step, so that the penalty applies to its answer
                    slot.prefill(history[:-1])
                    tok = slot.decode(history[-1], recent=history, repeat_penalty=repeat_penalty, repeat_last_n=repeat_last_n)
                else:
                    tok = slot.prefill(history)
                got = [tok]
                while len(got) < n:
                    history.append(tok)
                    tok = slot.decode(tok, recent=history if logits_penalised else None, repeat_penalty=repeat_penalty, repeat_last_n=repeat_last_n)
                    got.append(tok)
                out[i] = got
        except Exception as e:
            errors.append(e)

    threads = [threading.Thread(target=one, args=(i,)) for i in range(len(prompts))]
    for t in threads:
        t.start()
    for t in threads:
        t.join()
    pool.close()
    if errors:
        raise errors[0]
    return out


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv[:1] == ["trace"]:
        from .trace import main as trace_main

        return trace_main(argv[1:])
    if argv[:1] == ["build"]:
        from . import build

        build.build_all(force="--force" in argv, verbose="-v" in argv)
        return 0
    ap = argparse.ArgumentParser(prog="python -m orangu_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate")
    g.add_argument("--model", required=True, help=".gguf file, or a folder with config.json and model.safetensors")
    g.add_argument("--tokens", action="append", required=True, help="a prompt as token ids with commas between them; may be repeated")
    g.add_argument("--n", type=int, default=32, help="tokens to generate per prompt")
    g.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    g.add_argument("--max-seq-len", type=int, default=4096)
    g.add_argument("--repeat-penalty", type=float, default=1.0)
    g.add_argument("--repeat-last-n", type=int, default=64)
    sub.add_parser("trace")
    sub.add_parser("build")
    a = ap.parse_args(argv)

    from . import CudaBackend
    from .registry import load_model

    prompts = [[int(t) for t in p.split(",")] for p in a.tokens]
    backend = CudaBackend.init(0)
    model = load_model(backend, a.model, dtype=a.dtype, max_seq_len=a.max_seq_len, kv_pool_tokens=a.max_seq_len * len(prompts), state_slots=len(prompts))
    for got in generate(model, prompts, a.n, a.repeat_penalty, a.repeat_last_n):
        print(",".join(map(str, got)))
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
