#!/usr/bin/env python
"""Decode throughput of the quantized Llama-style hot path on B200, next to the CPU restatement.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl reference]

Workload (N = 1): random-init 8B-shape decoder in Q4_K_M (Q6_K for output and attn_v), 32 layers,
d_model 4096, 32 query / 8 KV heads of 128, FFN 14336, vocab 128256; one sequence with a 4096-token
context of uniformly random token ids (prefilled through the same library), then greedy decode at
batch 1.  A step is one decode step (one new token per sequence).  N > 1 runs the same model
tensor-parallel over N GPUs of one node (one process per GPU, NCCL all-reduce after the attention-output
and FFN-down products), so the total work is fixed: strong scaling.

One JSON line on stdout (rank 0):
  value      tokens/s over the K timed steps with the loop resident on the device (ob_decode_loop),
             device time from CUDA events, max over ranks
  e2e        the same metric through ob_decode_greedy, one host round trip per token: the token id and
             position go up from pinned host memory and the sampled id comes back, inside the timed region
  roofline   the dominant kernel (Q4_K single-token GEMV) run alone over every layer's Q4_K matrices,
             timed with CUDA events on its launching stream, against the measured HBM copy bandwidth
  cpu_baseline  the CPU restatement of the reference's path (oracle/) timed on this host's cores

--impl reference times that CPU path as the whole job.  The reference engine is Rust and there is no Rust
toolchain on these machines, so the arm runs oracle/, its line-by-line C++ restatement.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "tests"))  # tests/oracle.py: the ctypes binding of the CPU oracle

# torch.distributed.run exports OMP_NUM_THREADS=1; the synthetic-weight generator and the CPU oracle are OpenMP code and
# would take minutes on one thread.  Give every rank its share of the host cores (before any OpenMP runtime starts).
if int(os.environ.get("WORLD_SIZE", "1")) > 1 and os.environ.get("OMP_NUM_THREADS", "1") == "1":
    # the reference arm works on rank 0 alone (the other ranks return at once): it gets all the cores
    _ranks_at_work = 1 if "reference" in sys.argv else int(os.environ.get("LOCAL_WORLD_SIZE", os.environ["WORLD_SIZE"]))
    os.environ["OMP_NUM_THREADS"] = str(max(1, (os.cpu_count() or 1) // _ranks_at_work))

import numpy as np  # noqa: E402

METRIC = "decode tok/s (8B-shape Q4_K_M, bs1 & bs64); quantized GEMV HBM GB/s vs peak"
UNIT = "tok/s"
FALLBACK_HBM_GBS = 6650.0


def parse_args():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--model", default="8b", help="shape from orangu_b200.synth.CONFIGS")
    ap.add_argument("--layers", type=int, default=0, help="override the layer count (debugging only; invalidates the number)")
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--batch64-steps", type=int, default=16, help="steps of the 64-sequence decode measured as an extra (0 = skip)")
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--fenipel", default="", metavar="SIZE[,SIZE]", help="instead of the workload above: prefill and decode of Fenipel at these sizes "
                    "(1b, 8b; random weights) beside the quantized Llama shape of the same widths")
    ap.add_argument("--fenipel-layers", type=int, default=8, help="layers of both models in that comparison")
    ap.add_argument("--fenipel-only", action="store_true", help="leave the Llama shape out")
    ap.add_argument("--nenodra", default="", metavar="SIZE[,SIZE]", help="instead of the workload above: prefill and decode of Nenodra at these sizes "
                    "(1b, 8b; random weights) beside Fenipel at the same widths")
    ap.add_argument("--nenodra-layers", type=int, default=8, help="layers of both models in that comparison")
    ap.add_argument("--nenodra-only", action="store_true", help="leave Fenipel out")
    ap.add_argument("--senuvik", default="", metavar="SIZE[,SIZE]", help="instead of the workload above: prefill and decode of Senuvik at these sizes "
                    "(1b, 8b: widths) beside Nenodra at the same widths; one JSON line of its own")
    ap.add_argument("--senuvik-layers", type=int, default=8, help="layers of both models in that comparison")
    ap.add_argument("--senuvik-only", action="store_true", help="leave Nenodra out")
    ap.add_argument("--filorax", default="", metavar="SIZE[,SIZE]", help="instead of the workload above: prefill and decode of Filorax at these sizes "
                    "(1b, 8b: widths) beside Fenipel at the same widths; one JSON line of its own")
    ap.add_argument("--filorax-layers", type=int, default=8, help="layers of both models in that comparison")
    ap.add_argument("--filorax-only", action="store_true", help="leave Fenipel out")
    return ap.parse_args()


def measured_peak_gbs():
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            return float(json.load(f)["hbm_gbs"]), "measured"
    except Exception:
        return FALLBACK_HBM_GBS, "fallback"


# ---------------------------------------------------------------------------------------- clocks
class ClockSampler:
    """nvidia-smi clock / throttle-reason samples every 200 ms while a timed region runs."""

    FIELDS = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,clocks_event_reasons.hw_slowdown,"
              "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.gpu = gpu_index
        self.path = tempfile.mktemp(prefix="ob_clocks_", suffix=".csv")
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "200", "-i", str(self.gpu)],
                                         stdout=open(self.path, "w"), stderr=subprocess.DEVNULL)
        except OSError:
            self.proc = None

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.25)
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        sm, mx, reasons = [], [], set()
        try:
            for line in open(self.path):
                f = [x.strip() for x in line.split(",")]
                if len(f) < 9:
                    continue
                try:
                    sm.append(float(f[1]))
                    mx.append(float(f[2]))
                except ValueError:
                    continue
                for name, val in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"), f[5:9]):
                    if val.lower().startswith("active"):
                        reasons.add(name)
            os.unlink(self.path)
        except OSError:
            pass
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None, "reasons": sorted(reasons),
                "samples": len(sm)}


# ---------------------------------------------------------------------------------------- weights
def model_config(args):
    from orangu_b200 import synth

    cfg = dict(synth.CONFIGS[args.model])
    if args.layers:
        cfg["n_layer"] = args.layers
    return cfg


def build_tensors(cfg, rank: int, world: int, barrier):
    """Seeded synthetic tensors.  The generator is counter-based, so with several ranks every rank makes only its own
    tensor-parallel shards (the same bytes the whole tensors hold there) and hands them over as they are (tp_presliced)."""
    from orangu_b200 import synth

    return synth.model_tensors(cfg, seed=20240, tp=(rank, world) if world > 1 else None)


def algorithmic_bytes_per_token(cfg, context: int) -> int:
    """Quantized weight bytes every layer and the output projection read for one token, the f32 norm vectors,
    and the fp16 K/V of the attended window.  The embedding row and activations are not counted."""
    from orangu_b200.backend import tensor_byte_size

    e, hd = cfg["n_embd"], cfg["head_dim"]
    qd, kvd, ff, V = cfg["n_head"] * hd, cfg["n_head_kv"] * hd, cfg["n_ff"], cfg["n_vocab"]
    q4 = lambda o, i: o * tensor_byte_size(12, i)  # noqa: E731
    q6 = lambda o, i: o * tensor_byte_size(14, i)  # noqa: E731
    layer = q4(qd, e) + q4(kvd, e) + q6(kvd, e) + q4(e, qd) + 2 * q4(ff, e) + q4(e, ff) + 2 * e * 4
    return cfg["n_layer"] * layer + q6(V, e) + e * 4 + 2 * kvd * 2 * cfg["n_layer"] * context



# ---------------------------------------------------------------------------------------- single products (configs 1 and 2)
def operator_gemv_rooflines(be, peak):
    """The Backend::matmul operator at one token on device-resident buffers: BASELINE.json's single Q8_0 GEMV (4096 x 4096) and
    the Q4_K / Q6_K sweep shapes.  A single product moves 10-50 MB -- a few microseconds -- so it is timed inside a CUDA graph
    of `reps` back-to-back launches; the launches rotate over enough copies of the matrix to exceed the 126 MB L2, so every
    launch reads its weights from HBM.  Algorithmic bytes = GGUF bytes of the matrix + the fp32 input and output vectors."""
    import torch

    from orangu_b200 import QuantMatrix, capi, synth
    from orangu_b200.backend import tensor_byte_size

    L = capi.load()
    out = {}
    cases = [("config 1: Q8_0 4096x4096", 8, 4096, 4096)] + [
        (f"config 2: {'Q4_K' if t == 12 else 'Q6_K'} {o}x{i}", t, o, i) for t in (12, 14) for (o, i) in ((4096, 4096), (14336, 4096), (4096, 14336))]
    stream = torch.cuda.Stream()
    for name, t, out_dim, in_dim in cases:
        wbytes = out_dim * tensor_byte_size(t, in_dim)
        copies = max(2, -(-160_000_000 // wbytes))
        mats = [synth.matrix(t, out_dim, in_dim, 900 + c) for c in range(copies)]
        handles = [be._weight(QuantMatrix(m["data"], t, in_dim, out_dim)) for m in mats]
        x = torch.randn(in_dim, device="cuda", dtype=torch.float32)
        y = torch.empty(out_dim, device="cuda", dtype=torch.float32)
        reps = 4 * copies
        with torch.cuda.stream(stream):
            for h in handles:  # warm-up outside capture: scratch allocation, one-time kernel attributes
                capi.check(be._h, L.ob_matmul_device(be._h, x.data_ptr(), 1, h, y.data_ptr(), 0, stream.cuda_stream))
            stream.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=stream):
                for r in range(reps):
                    capi.check(be._h, L.ob_matmul_device(be._h, x.data_ptr(), 1, handles[r % copies], y.data_ptr(), 0, stream.cuda_stream))
            g.replay()
            stream.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(stream)
            for _ in range(5):
                g.replay()
            e1.record(stream)
            stream.synchronize()
        us = e0.elapsed_time(e1) * 1e3 / (5 * reps)
        nbytes = wbytes + 4 * (in_dim + out_dim)
        out[name] = {"avg_launch_us": us, "algorithmic_bytes": nbytes, "GB/s": nbytes / us / 1e3, "frac": nbytes / us / 1e3 / peak,
                     "timed": f"CUDA graph of {reps} products rotating over {copies} copies of the matrix ({copies * wbytes / 1e6:.0f} MB > L2), 5 replays",
                     "kernels_per_product": 1}
        for h in handles:
            L.ob_weight_release(be._h, h)
            be._weights.remove(h)
    return out


# ---------------------------------------------------------------------------------------- 70B shape under tensor parallel
def run_70b(be, rank, world, uid, barrier, max_over_ranks, peak):
    """BASELINE.json's last configuration: 70B-shape Q4_K_M decoder (80 layers, d_model 8192, 64 query / 8 KV heads, FFN 28672),
    tensor parallel over this run's GPUs, batch-1 and batch-32 greedy decode at an 8192-token context.  Every rank generates
    only its own shards.  Reports tokens/s (device time, max over ranks) and the per-GPU fraction of the HBM roofline."""
    import orangu_b200
    from orangu_b200 import synth

    cfg = dict(synth.CONFIGS["70b"])
    ctx_len, steps1, steps32, n_seq = 8192, 8, 4, 32
    t0 = time.time()
    tensors = synth.model_tensors(cfg, seed=20270, tp=(rank, world))
    t_gen = time.time() - t0
    per_seq = ctx_len + 64
    model = orangu_b200.LlamaModel(be, cfg, tensors, max_seq_len=per_seq, max_batch_tokens=512, kv_pool_tokens=n_seq * per_seq + 64,
                                   tp_rank=rank, tp_size=world, tp_unique_id=uid, tp_presliced=True)
    del tensors
    kv = model.new_kv_cache(per_seq)
    prompt = np.random.default_rng(13).integers(0, cfg["n_vocab"], ctx_len).astype(np.uint32)
    t0 = time.time()
    first = model.forward_maybe_sampling(kv, prompt, 0)
    t_prefill = time.time() - t0
    model.decode_loop([kv], [first], 3)
    barrier()
    model.decode_loop([kv], [int(first)], steps1)
    ms1 = max_over_ranks(be.last_device_ms()) / steps1
    kv.truncate(ctx_len)
    caches = [kv]
    for _ in range(n_seq - 1):
        c = model.new_kv_cache(per_seq)
        c.copy_prefix_from(kv, ctx_len)
        caches.append(c)
    firsts = [int(first)] * n_seq
    model.decode_loop(caches, firsts, 2)
    barrier()
    model.decode_loop(caches, firsts, steps32)
    ms32 = max_over_ranks(be.last_device_ms()) / steps32
    w_bytes = algorithmic_bytes_per_token(cfg, 0)
    kv_bytes = algorithmic_bytes_per_token(cfg, ctx_len) - w_bytes
    out = {"workload": "70B-shape Llama decoder, Q4_K_M (Q6_K output and attn_v), 80 layers, context 8192 prefilled through the library",
           "parallelism": f"tp{world}", "setup_s": {"synthetic_shards": round(t_gen, 1), "prefill_8192": round(t_prefill, 1)},
           "batch1": {"value": 1e3 / ms1, "unit": UNIT, "ms_per_step": ms1, "steps": steps1,
                      "hbm_frac_per_gpu": (w_bytes + kv_bytes) / world / (ms1 * 1e-3) / 1e9 / peak},
           "batch32": {"value": n_seq * 1e3 / ms32, "unit": UNIT, "ms_per_step": ms32, "steps": steps32, "sequences": n_seq,
                       "kv": "31 sequences share the first one's prefilled pages by device copy (KvCache::copy_prefix_from)",
                       "hbm_frac_per_gpu": (w_bytes + n_seq * kv_bytes) / world / (ms32 * 1e-3) / 1e9 / peak}}
    model.close()
    return out

# ---------------------------------------------------------------------------------------- CPU arm
def cpu_decode_tokens_per_s(cfg, tensors, budget_s: float, max_tokens: int):
    """Times greedy decode of the CPU oracle on all host cores.  Bounded: a short prompt (the CPU prefill of a
    4096-token context would take minutes), then as many single-token steps as fit the budget."""
    import oracle as O

    ref = O.Model(cfg, tensors)
    cores = O.hardware_threads()
    prompt = np.random.default_rng(7).integers(0, cfg["n_vocab"], 4).astype(np.uint32)
    kv = ref.new_kv(4 + max_tokens + 2, f16=True)
    tok = O.argmax(ref.forward(kv, prompt, 0))
    tok = O.argmax(ref.forward(kv, [tok], 4))  # one untimed step: page the weights in
    n, t0 = 0, time.perf_counter()
    while n < max_tokens:
        tok = O.argmax(ref.forward(kv, [tok], 5 + n))
        n += 1
        if time.perf_counter() - t0 > budget_s:
            break
    dt = time.perf_counter() - t0
    return n / dt, cores, f"{n} greedy decode steps at batch 1 after a 4-token prompt (context {5}..{5 + n}), {dt:.1f} s, OpenMP over output rows"


def run_reference(args, rank: int, world: int):
    """The reference arm: the reference's CPU path (its C++ restatement under oracle/) as the whole job."""
    if rank != 0:
        return
    from orangu_b200 import synth  # noqa: F401  (the synthetic tensors are shared with our arm)

    cfg = model_config(args)
    tensors = build_tensors(cfg, 0, 1, lambda: None)
    import oracle as O

    ref = O.Model(cfg, tensors)
    cores = O.hardware_threads()
    prompt = np.random.default_rng(7).integers(0, cfg["n_vocab"], 4).astype(np.uint32)
    kv = ref.new_kv(8 + args.warmup + args.steps, f16=True)
    tok = O.argmax(ref.forward(kv, prompt, 0))
    pos = 4
    for _ in range(args.warmup):
        tok = O.argmax(ref.forward(kv, [tok], pos))
        pos += 1
    t0 = time.perf_counter()
    for _ in range(args.steps):
        tok = O.argmax(ref.forward(kv, [tok], pos))
        pos += 1
    dt = time.perf_counter() - t0
    value = args.steps / dt
    sample = (f"{args.steps} greedy decode steps at batch 1 after a 4-token prompt; the 4096-token context is not prefilled on the CPU "
              f"(its attention share at that length is under 10% of a step)")
    line = {
        "impl": "reference", "metric": METRIC, "value": value, "unit": UNIT, "n_gpus": args.gpus, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": dt / args.steps * 1e3, "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "int8", "data": "synthetic",
        "config": {"workload": f"{args.model}-shape Q4_K_M decode, batch 1, CPU path of the reference restated in C++ (oracle/); no Rust toolchain here",
                   "n_layer": cfg["n_layer"], "host_cores": cores, "context": f"{4 + args.warmup}..{4 + args.warmup + args.steps} positions (a 4-token prompt; the GPU arm decodes at {args.context})"},
        "cpu_baseline": {"value": value, "unit": UNIT, "cores": cores, "kind": "port", "sample": sample},
        "e2e": {"value": value, "unit": UNIT, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "gpu_launches": 0,
    }
    print(json.dumps(line), flush=True)


# ---------------------------------------------------------------------------------------- our arm
FENIPEL_SIZES = {  # widths and feed-forwards of the Llama shapes of the same name; half of the layers attend, half retain
    "1b": {"width": 2048, "ff": 8192, "vocab": 32768, "side": 128,
           "latent": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 384, "window": 1024},
           "retention": {"heads": 8, "dim": 128, "vdim": 256}},
    "8b": {"width": 4096, "ff": 14336, "vocab": 32768, "side": 256,
           "latent": {"heads": 32, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "window": 1024},
           "retention": {"heads": 16, "dim": 128, "vdim": 256}},
}


def random_matrices():
    """lin(rows, columns): bfloat16 bits of normal values over the root of the columns (or times std), all dealt out from one pool."""
    import numpy as np
    from orangu_b200.safetensors import to_bf16

    pool = np.random.default_rng(1).normal(size=1 << 22).astype(np.float32)
    cache, turn = {}, [0]

    def lin(o, i, std=None):
        std = i ** -0.5 if std is None else std
        if std not in cache:
            cache[std] = to_bf16(pool * std)
        bits = cache[std]
        turn[0] += 1
        return np.resize(np.roll(bits, (turn[0] * 104729) % bits.size), (o, i))

    return lin


def fenipel_model(size: str, n_layer: int):
    """Configuration and random bfloat16 tensors (bits)."""
    import numpy as np
    from orangu_b200.safetensors import to_bf16

    z = FENIPEL_SIZES[size]
    E, V, sd = z["width"], z["vocab"], z["side"]
    lin = random_matrices()
    layers, t = [], {"embed": lin(V, E), "head": lin(V, E), "final.norm": to_bf16(np.float32(1)), "side.embed": lin(V, n_layer * sd)}
    for n in range(n_layer):
        at, m = f"l{n}.mix.", dict(z["latent" if n % 2 == 0 else "retention"])
        H, d, v = m["heads"], m["dim"], m["vdim"]
        if n % 2 == 0:
            R, K = m["rot_dim"], m["kv_rank"]
            m.update(mask={"size": m.pop("window")}, rot={"base": 10000.0, "dims": R}, scale=(d + R) ** -0.5)
            t.update({at + "q": lin(H * (d + R), E), at + "dkv": lin(K + R, E), at + "dkv.norm": to_bf16(np.ones(K)), at + "uk": lin(H * d, K), at + "uv": lin(H * v, K),
                      at + "g": lin(H, E)})
        else:
            m.update(rot={"base": 10000.0, "dims": d}, decay=[1 - 2.0 ** (-5 - 0.5 * h) for h in range(H)])
            t.update({at + "q": lin(H * d, E), at + "k": lin(H * d, E), at + "v": lin(H * v, E), at + "g": lin(H * v, E)})
        t.update({at + "o": lin(E, H * v), f"l{n}.norm1": to_bf16(np.float32(1)), f"l{n}.mlp.gate": lin(z["ff"], E), f"l{n}.mlp.up": lin(z["ff"], E),
                  f"l{n}.mlp.down": lin(E, z["ff"]), f"l{n}.side.gate": lin(sd, E), f"l{n}.side.proj": lin(E, sd), f"l{n}.side.norm": to_bf16(np.ones(E))})
        layers.append({"type": "latent_attention" if n % 2 == 0 else "retention", "mixer": m, "mlp": {"kind": "dense", "ff": z["ff"], "limit": 7.0}})
    return {"architecture": "Fenipel", "vocab": V, "width": E, "norm": {"eps": 1e-6}, "token_side": {"dim": sd}, "layers": layers}, t


NENODRA_SIZES = {  # Fenipel's widths; half of the layers have two maps and a dense feed-forward, half are gated with experts
    "1b": {"width": 2048, "ff": 8192, "vocab": 32768, "experts": 16, "top": 2, "expert_ff": 1024,
           "attention": {"heads": 16, "kv_heads": 4, "dim": 64, "vdim": 128, "diff": 0.5}, "attention_2": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128}, "window": 1024},
    "8b": {"width": 4096, "ff": 14336, "vocab": 32768, "experts": 16, "top": 2, "expert_ff": 2048,
           "attention": {"heads": 32, "kv_heads": 8, "dim": 64, "vdim": 128, "diff": 0.5}, "attention_2": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128}, "window": 1024},
}


def nenodra_model(size: str, n_layer: int):
    """Configuration and random bfloat16 tensors (bits)."""
    import numpy as np
    from orangu_b200.safetensors import to_bf16

    z = NENODRA_SIZES[size]
    E, V = z["width"], z["vocab"]
    lin, const = random_matrices(), lambda v, n: to_bf16(np.full(n, v, np.float32))
    layers, t = [], {"embed": lin(V, E, 4.0), "head": lin(V, E), "final.norm": const(0, E)}  # (tokens differ enough to choose different experts)
    for n in range(n_layer):
        kind = "attention" if n % 2 == 0 else "attention_2"
        at, m = f"l{n}.mix.", dict(z[kind], mask={"size": z["window"]})
        H, G, d, v, maps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], 2 - n % 2
        m.update(rot={"base": 10000.0, "dims": d}, scale=d ** -0.5)
        t.update({at + "q": lin(H * maps * d, E), at + "k": lin(G * maps * d, E), at + "q.norm": const(1, d), at + "k.norm": const(1, d), at + "o": lin(E, H * v),
                  f"l{n}.norm1": const(0, E), f"l{n}.norm2": const(0, E)})
        if maps == 2:
            t.update({at + "v": lin(G * v, E), at + "q.b": const(0.1, H * 2 * d), at + "k.b": const(0.1, G * 2 * d), at + "v.b": const(0.1, G * v), at + "o.b": const(0.1, E)})
            t.update({at + x: const(0.05, d) for x in ("lq1", "lk1", "lq2", "lk2")})
            t.update({f"l{n}.mlp.up": lin(z["ff"], E), f"l{n}.mlp.down": lin(E, z["ff"])})
            mlp = {"kind": "dense", "ff": z["ff"]}
        else:
            X, ff = z["experts"], z["expert_ff"]
            t.update({at + "g": lin(H * v, E), f"l{n}.mlp.router": lin(X, E)})
            for e in range(X):
                t.update({f"l{n}.mlp.e{e}.gate": lin(ff, E), f"l{n}.mlp.e{e}.up": lin(ff, E), f"l{n}.mlp.e{e}.down": lin(E, ff)})
            mlp = {"kind": "moe", "router": {"experts": X, "top": z["top"]}, "expert": {"ff": ff}}
        layers.append({"type": kind, "mixer": m, "mlp": mlp})
    return {"architecture": "Nenodra", "vocab": V, "width": E, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "logit_scale": 1.0, "layers": layers}, t


SENUVIK_SIZES = {  # Nenodra's widths, heads and experts; of four layers one attends within a window (dense), two are parallel, one is a state space
    "1b": {"width": 2048, "ff": 8192, "vocab": 32768, "experts": 16, "top": 2, "expert_ff": 1024, "window": 1024, "keep": 4,
           "attention": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128}, "space": {"heads": 64, "vdim": 64, "state": 128, "groups": 4, "norm_groups": 4, "conv": 4},
           "time": {"heads": 32, "dim": 64}, "rank": 64},
    "8b": {"width": 4096, "ff": 14336, "vocab": 32768, "experts": 16, "top": 2, "expert_ff": 2048, "window": 1024, "keep": 4,
           "attention": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128}, "space": {"heads": 128, "vdim": 64, "state": 128, "groups": 8, "norm_groups": 8, "conv": 4},
           "time": {"heads": 64, "dim": 64}, "rank": 128},
}


def senuvik_model(size: str, n_layer: int):
    """Configuration and random bfloat16 tensors (bits)."""
    import numpy as np
    from orangu_b200.safetensors import to_bf16

    z = SENUVIK_SIZES[size]
    E, V = z["width"], z["vocab"]
    lin, const = random_matrices(), lambda v, *n: to_bf16(np.full(n, v, np.float32))
    layers, t = [], {"embed": lin(V, E, 4.0), "head": lin(V, E), "final.norm": const(1, E)}  # (tokens differ enough to choose different experts)
    a = z["attention"]
    H, G, d, v = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
    for n in range(n_layer):
        kind = ("attention", "parallel", "mamba2", "parallel")[n % 4]
        at = f"l{n}.mix."
        t.update({f"l{n}.{x}": const(1, E) for x in ("norm1", "norm2", "norm1b", "norm2b", "ls1", "ls2")})
        if kind == "attention":
            mixer = dict(a, mask={"size": z["window"], "keep_first": z["keep"]}, rot={"base": 10000.0, "dims": d, "scaling": {"factor": 4.0}}, scale=d ** -0.5)
            t.update({at + "q": lin(H * d, E), at + "q.b": const(0.1, H * d), at + "q.norm": const(1, H * d), at + "k": lin(G * d, E), at + "k.b": const(0.1, G * d),
                      at + "k.norm": const(1, G * d), at + "v": lin(G * v, E), at + "v.b": const(0.1, G * v), at + "sink": const(0.5, H), at + "o": lin(E, H * v)})
        elif kind == "mamba2":
            mixer = s = dict(z["space"])
            inner = s["heads"] * s["vdim"]
            ch = inner + 2 * s["groups"] * s["state"]
            t.update({at + "in": lin(inner + ch + s["heads"], E), at + "conv": lin(ch, s["conv"]), at + "conv.b": const(0.1, ch), at + "dt_bias": const(-2, s["heads"]),
                      at + "A_log": const(0.5, s["heads"]), at + "D": const(1, s["heads"]), at + "norm": const(1, inner), at + "o": lin(E, inner)})
        else:
            r, m = z["time"], z["time"]["heads"] * z["time"]["dim"]
            mixer = {"left": dict(a, rot={"base": 1e6, "dims": d, "scaling": {"factor": 4.0, "original": 1024, "fast": 32.0, "slow": 1.0}}, scale=d ** -0.5, softcap=50.0),
                     "right": dict(r), "left_scale": 1.0, "right_scale": 1.0}
            t.update({at + "left.q": lin(H * d, E), at + "left.k": lin(G * d, E), at + "left.v": lin(G * v, E), at + "left.g": lin(H, E), at + "left.o": lin(E, H * v)})
            t.update({at + "right." + c: lin(m, E) for c in "rkvg"})
            t.update({at + "right.mu." + c: const(0.5, E) for c in "rkvgw"})
            t.update({at + "right.w1": lin(z["rank"], E), at + "right.w2": lin(m, z["rank"]), at + "right.w0": const(-3, m), at + "right.u": const(0.5, r["heads"], r["dim"]),
                      at + "right.norm": const(1, m), at + "right.o": lin(E, m)})
        if n % 4 == 0:
            mlp = {"kind": "dense", "ff": z["ff"]}
            t.update({f"l{n}.mlp.gate": lin(z["ff"], E), f"l{n}.mlp.up": lin(z["ff"], E), f"l{n}.mlp.down": lin(E, z["ff"])})
        else:
            X, ff = z["experts"], z["expert_ff"]
            mlp = {"kind": "moe", "router": {"experts": X, "top": z["top"]}, "expert": {"ff": ff}, "shared": {"ff": ff}}
            t.update({f"l{n}.mlp.router": lin(X, E), f"l{n}.mlp.shared.sg": lin(1, E)})
            for e in [f"e{e}." for e in range(X)] + ["shared."]:
                t.update({f"l{n}.mlp.{e}gate": lin(ff, E), f"l{n}.mlp.{e}up": lin(ff, E), f"l{n}.mlp.{e}down": lin(E, ff)})
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Senuvik", "vocab": V, "width": E, "norm": {"eps": 1e-6}, "layers": layers}, t


FILORAX_SIZES = {  # Fenipel's widths, heads and latents, Senuvik's experts; two layers of three attend within a window, one is causal and rotated
    "1b": {"width": 2048, "vocab": 32768, "experts": 16, "top": 2, "groups": 4, "keep": 2, "expert_ff": 1024, "taps": 4, "norm_groups": 8,
           "latent": {"heads": 16, "dim": 128, "vdim": 128, "kv_rank": 384}, "rot_dim": 64, "windows": (512, 1024)},
    "8b": {"width": 4096, "vocab": 32768, "experts": 16, "top": 2, "groups": 4, "keep": 2, "expert_ff": 2048, "taps": 4, "norm_groups": 16,
           "latent": {"heads": 32, "dim": 128, "vdim": 128, "kv_rank": 512}, "rot_dim": 64, "windows": (512, 1024)},
}


def filorax_model(size: str, n_layer: int):
    """Configuration and random bfloat16 tensors (bits)."""
    import numpy as np
    from orangu_b200.safetensors import to_bf16

    z = FILORAX_SIZES[size]
    E, V, X, ff, taps = z["width"], z["vocab"], z["experts"], z["expert_ff"], z["taps"]
    lin, const = random_matrices(), lambda v, *n: to_bf16(np.full(n, v, np.float32))
    layers, t = [], {"embed": lin(V, E, 4.0), "head": lin(V, E), "final.norm": const(1, E)}  # (tokens differ enough to choose different experts)
    for n in range(n_layer):
        kind = ("latent_attention_3", "latent_attention", "latent_attention_2")[n % 3]
        at, m = f"l{n}.mix.", dict(z["latent"])
        H, d, v, K = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        R = z["rot_dim"] if n % 3 == 2 else 0
        m.update(scale=(d + R) ** -0.5)
        m.update({"rot_dim": R, "rot": {"base": 10000.0, "dims": R}} if R else {"mask": {"size": z["windows"][n % 3]}})
        t.update({at + "q": lin(H * (d + R), E), at + "dkv": lin(K + R, E), at + "dkv.norm": const(1, K), at + "uk": lin(H * d, K), at + "uv": lin(H * v, K), at + "o": lin(E, H * v)})
        if n % 3:
            t.update({at + "sink": const(0.5, H), at + "g": lin(H * v, E)})
        t.update({f"l{n}.norm1": const(1, E), f"l{n}.norm2": const(1, E), f"l{n}.canon1": lin(E, taps, 0.25), f"l{n}.canon2": lin(E, taps, 0.25), f"l{n}.dwa": const(1 / (n + 2), n + 2)})
        t.update({f"l{n}.mlp.router": lin(X, E), f"l{n}.mlp.shared.sg": lin(1, E)})
        for e in [f"e{e}." for e in range(X)] + ["shared."]:
            t.update({f"l{n}.mlp.{e}gate": lin(ff, E), f"l{n}.mlp.{e}up": lin(ff, E), f"l{n}.mlp.{e}down": lin(E, ff)})
        router = {"experts": X, "top": z["top"], "scale": 1.0, "groups": {"count": z["groups"], "keep": z["keep"]}}
        layers.append({"type": kind, "mixer": m, "mlp": {"kind": "moe", "router": router, "expert": {"ff": ff}, "shared": {"ff": ff}}})
    return {"architecture": "Filorax", "vocab": V, "width": E, "norm": {"eps": 1e-6, "groups": z["norm_groups"]}, "canon": {"taps": taps}, "residual_mult": 1.0,
            "layers": layers}, t


def time_model(be, model, vocab: int, weight_bytes, cache_bytes_per_token: float, flops_per_token: float, steps: int, warmup: int, prompt: int = 4096):
    """Prefill of one prompt and greedy decode loops at batch 1, 8 and 64 (device time, CUDA events; weights exceed L2).
    weight_bytes: read per decoded step, a number or a function of the batch.  cache_bytes_per_token: cache and state traffic of
    one decoded token at this context."""
    import numpy as np

    rng = np.random.default_rng(0)
    toks = rng.integers(0, vocab, prompt)
    peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json"))) if os.path.exists(os.path.join(ROOT, "MEASURED_PEAKS.json")) else {}
    hbm, tf = peaks.get("hbm_gbs", 6650.0), peaks.get("bf16_tflops_sustained", 1400.0)
    out = {"decode": {}}
    room = prompt + 4 * (steps + warmup)
    kv, ms = model.new_kv_cache(room, paged=True), []
    for _ in range(4):
        kv.truncate(0)
        model.forward_maybe_sampling(kv, toks, 0)
        ms.append(be.last_device_ms())
    best = min(ms[1:])
    out["prefill"] = {"tokens": prompt, "ms": best, "tok_s": prompt / best * 1e3, "of_bf16_sustained": prompt * flops_per_token / (best * 1e-3) / (tf * 1e12)}
    kvs = [kv]
    for batch in (1, 8, 64):
        while len(kvs) < batch:
            k = model.new_kv_cache(room, paged=True)
            k.copy_prefix_from(kv, len(kv))
            kvs.append(k)
        first = [int(x) for x in rng.integers(0, vocab, batch)]
        model.decode_loop(kvs[:batch], first, warmup)
        model.decode_loop(kvs[:batch], first, steps)
        t = be.last_device_ms() / steps
        need = (weight_bytes(batch) if callable(weight_bytes) else weight_bytes) + batch * cache_bytes_per_token
        out["decode"][str(batch)] = {"ms_per_step": t, "tok_s": batch / t * 1e3, "bytes_per_step": need, "of_hbm": need / (t * 1e-3) / (hbm * 1e9)}
    for k in kvs:
        k.close()
    return out


def time_fenipel(be, size: str, L: int, steps: int, warmup: int):
    import orangu_b200

    cfg, t = fenipel_model(size, L)
    n = sum(a.size for k, a in t.items() if not k.endswith("embed"))
    z, prompt = FENIPEL_SIZES[size], 4096
    la, re = z["latent"], z["retention"]
    win = min(la["window"], prompt)
    n_lat, n_ret = (L + 1) // 2, L // 2
    cache = n_lat * win * (la["kv_rank"] + la["rot_dim"]) * 2 + n_ret * re["heads"] * re["dim"] * re["vdim"] * 8
    flops = 2 * n + n_lat * 2 * win * la["heads"] * (la["dim"] + la["rot_dim"] + la["vdim"]) + n_ret * 4 * re["heads"] * re["dim"] * re["vdim"]
    m = orangu_b200.FenipelModel(be, cfg, t, max_seq_len=8192, max_batch_tokens=prompt, kv_pool_tokens=64 * 4480, state_slots=64)
    result = dict(time_model(be, m, z["vocab"], 2 * n, cache, flops, steps, warmup), parameters=n)
    m.close()
    return result


def time_nenodra(be, size: str, L: int, steps: int, warmup: int):
    import orangu_b200

    cfg, t = nenodra_model(size, L)
    z, prompt = NENODRA_SIZES[size], 4096
    expert = 3 * z["width"] * z["expert_ff"]
    n_moe = sum(x["mlp"]["kind"] == "moe" for x in cfg["layers"])
    n = sum(a.size for k, a in t.items() if not k.endswith("embed"))
    shared = n - n_moe * z["experts"] * expert
    win, cache, flops = min(z["window"], prompt), 0, 2 * (shared + n_moe * z["top"] * expert)
    for layer in cfg["layers"]:
        m, maps = layer["mixer"], 2 if layer["type"] == "attention" else 1
        cache += 2 * win * m["kv_heads"] * (maps * m["dim"] + m["vdim"])
        flops += 2 * win * m["heads"] * maps * (m["dim"] + m["vdim"])
    # experts that a step reads when tokens choose independently and evenly
    weights = lambda batch: 2 * (shared + n_moe * expert * z["experts"] * (1 - (1 - z["top"] / z["experts"]) ** batch))
    m = orangu_b200.NenodraModel(be, cfg, t, max_seq_len=8192, max_batch_tokens=prompt, kv_pool_tokens=64 * 4480)
    result = dict(time_model(be, m, z["vocab"], weights, cache, flops, steps, warmup), parameters=n)
    m.close()
    return result


def time_senuvik(be, size: str, L: int, steps: int, warmup: int):
    import orangu_b200

    cfg, t = senuvik_model(size, L)
    z, prompt = SENUVIK_SIZES[size], 4096
    expert = 3 * z["width"] * z["expert_ff"]
    n_moe = sum(x["mlp"]["kind"] == "moe" for x in cfg["layers"])
    n = sum(a.size for k, a in t.items() if not k.endswith("embed"))
    every = n - n_moe * z["experts"] * expert
    a, s, r = z["attention"], z["space"], z["time"]
    cache, flops = 0, 2 * (every + n_moe * z["top"] * expert)
    for layer in cfg["layers"]:
        if layer["type"] == "mamba2":
            state = s["heads"] * s["state"] * s["vdim"]
            cache, flops = cache + 8 * state, flops + 6 * state
            continue
        seen = min(z["window"], prompt) if layer["type"] == "attention" else prompt
        cache += 2 * seen * a["kv_heads"] * (a["dim"] + a["vdim"])
        flops += 2 * (seen if layer["type"] == "attention" else prompt // 2) * a["heads"] * (a["dim"] + a["vdim"])
        if layer["type"] == "parallel":
            state = r["heads"] * r["dim"] ** 2
            cache, flops = cache + 8 * state, flops + 6 * state
    # experts that a step reads when tokens choose independently and evenly
    weights = lambda batch: 2 * (every + n_moe * expert * z["experts"] * (1 - (1 - z["top"] / z["experts"]) ** batch))
    m = orangu_b200.SenuvikModel(be, cfg, t, max_seq_len=8192, max_batch_tokens=prompt, kv_pool_tokens=64 * 4480, state_slots=64)
    result = dict(time_model(be, m, z["vocab"], weights, cache, flops, steps, warmup), parameters=n)
    m.close()
    return result


def time_filorax(be, size: str, L: int, steps: int, warmup: int):
    import orangu_b200

    cfg, t = filorax_model(size, L)
    z, prompt = FILORAX_SIZES[size], 4096
    expert = 3 * z["width"] * z["expert_ff"]
    n = sum(a.size for k, a in t.items() if not k.endswith("embed"))
    every = n - L * z["experts"] * expert
    cache, flops = L * 2 * (z["taps"] - 1) * z["width"] * 8, 2 * (every + L * z["top"] * expert)  # (last inputs of both sublayers, read and written)
    for layer in cfg["layers"]:
        m = layer["mixer"]
        R, win = m.get("rot_dim", 0), min(m["mask"]["size"], prompt) if "mask" in m else 0
        cache += 2 * (win or prompt) * (m["kv_rank"] + R)
        flops += 2 * (win or prompt // 2) * m["heads"] * (m["dim"] + R + m["vdim"])
    # experts that a step reads when tokens choose independently and evenly
    weights = lambda batch: 2 * (every + L * expert * z["experts"] * (1 - (1 - z["top"] / z["experts"]) ** batch))
    m = orangu_b200.FiloraxModel(be, cfg, t, max_seq_len=8192, max_batch_tokens=prompt, kv_pool_tokens=64 * 4480, state_slots=64)
    result = dict(time_model(be, m, z["vocab"], weights, cache, flops, steps, warmup), parameters=n)
    m.close()
    return result


def run_filorax(args):
    """--filorax: one JSON line with both models at every size."""
    import orangu_b200

    be = orangu_b200.CudaBackend.init(0)
    steps, warmup, L = args.steps, max(3, args.warmup), args.filorax_layers
    result = {"bench": "filorax", "data": "synthetic", "dtype": "bf16", "layers": L, "steps": steps, "warmup": warmup, "sizes": {}}
    clocks = ClockSampler(0)
    clocks.start()
    for size in args.filorax.split(","):
        entry = {"filorax": time_filorax(be, size, L, steps, warmup)}
        if not args.filorax_only:
            entry["fenipel"] = time_fenipel(be, size, L, steps, warmup)
        result["sizes"][size] = entry
    result["clocks"] = clocks.stop()
    be.close()
    print(json.dumps(result))


def run_senuvik(args):
    """--senuvik: one JSON line with both models at every size."""
    import orangu_b200

    be = orangu_b200.CudaBackend.init(0)
    steps, warmup, L = args.steps, max(3, args.warmup), args.senuvik_layers
    result = {"bench": "senuvik", "data": "synthetic", "dtype": "bf16", "layers": L, "steps": steps, "warmup": warmup, "sizes": {}}
    clocks = ClockSampler(0)
    clocks.start()
    for size in args.senuvik.split(","):
        entry = {"senuvik": time_senuvik(be, size, L, steps, warmup)}
        if not args.senuvik_only:
            entry["nenodra"] = time_nenodra(be, size, L, steps, warmup)
        result["sizes"][size] = entry
    result["clocks"] = clocks.stop()
    be.close()
    print(json.dumps(result))


def run_nenodra(args):
    """--nenodra: one JSON line with both models at every size."""
    import orangu_b200

    be = orangu_b200.CudaBackend.init(0)
    steps, warmup, L = args.steps, max(3, args.warmup), args.nenodra_layers
    result = {"bench": "nenodra", "data": "synthetic", "dtype": "bf16", "layers": L, "steps": steps, "warmup": warmup, "sizes": {}}
    clocks = ClockSampler(0)
    clocks.start()
    for size in args.nenodra.split(","):
        entry = {"nenodra": time_nenodra(be, size, L, steps, warmup)}
        if not args.nenodra_only:
            entry["fenipel"] = time_fenipel(be, size, L, steps, warmup)
        result["sizes"][size] = entry
    result["clocks"] = clocks.stop()
    be.close()
    print(json.dumps(result))


def run_fenipel(args):
    """--fenipel: one JSON line with both models at every size.  bf16 weights against Q4_K_M: equal parameter counts are not
    equal bytes, so fractions of the roofline are what compares."""
    import orangu_b200
    from orangu_b200 import synth

    be = orangu_b200.CudaBackend.init(0)
    steps, warmup, L = args.steps, max(3, args.warmup), args.fenipel_layers
    result = {"bench": "fenipel", "data": "synthetic", "dtype": "bf16", "layers": L, "steps": steps, "warmup": warmup, "sizes": {}}
    clocks = ClockSampler(0)
    clocks.start()
    for size in args.fenipel.split(","):
        entry = {"fenipel": time_fenipel(be, size, L, steps, warmup)}
        z, prompt = FENIPEL_SIZES[size], 4096
        if not args.fenipel_only:
            c = dict(synth.CONFIGS[size], n_layer=L, n_vocab=z["vocab"])
            tensors = synth.model_tensors(c, seed=7)
            wb = sum(x["data"].nbytes for k, x in tensors.items() if not k.startswith("token_embd"))
            elems = sum(x["in_dim"] * x["out_dim"] for k, x in tensors.items() if not k.startswith("token_embd") and "norm" not in k)
            kvd = c["n_head_kv"] * c["head_dim"]
            m = orangu_b200.LlamaModel(be, c, tensors, max_seq_len=8192, max_batch_tokens=512, kv_pool_tokens=64 * 4480)
            fl = 2 * elems + L * 2 * (prompt / 2) * c["n_head"] * c["head_dim"] * 2
            entry["llama_q4km"] = dict(time_model(be, m, z["vocab"], wb, L * prompt * kvd * 4, fl, steps, warmup), parameters=elems)
            m.close()
            del tensors
        result["sizes"][size] = entry
    result["clocks"] = clocks.stop()
    be.close()
    print(json.dumps(result))


def main():
    args = parse_args()
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if args.impl == "reference":
        run_reference(args, rank, world)
        return
    if args.fenipel:
        run_fenipel(args)
        return
    if args.senuvik:
        run_senuvik(args)
        return
    if args.filorax:
        run_filorax(args)
        return
    if args.nenodra:
        run_nenodra(args)
        return

    import torch
    import torch.distributed as dist

    import orangu_b200
    from orangu_b200 import capi

    if not torch.cuda.is_available():
        raise SystemExit("bench.py needs a CUDA device: there is no CPU fallback")
    torch.cuda.set_device(local_rank)
    if world > 1:
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        dist.init_process_group("nccl", device_id=torch.device("cuda", local_rank))

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    def max_over_ranks(x: float) -> float:
        if world == 1:
            return x
        t = torch.tensor([x], dtype=torch.float64, device="cuda")
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t.item())

    cfg = model_config(args)
    t_build = time.time()
    tensors = build_tensors(cfg, rank, world, barrier)
    t_build = time.time() - t_build

    be = orangu_b200.CudaBackend.init(local_rank)

    def make_uid():
        """A fresh communicator id from rank 0, the same 128 bytes on every rank."""
        if world == 1:
            return None
        buf = torch.zeros(128, dtype=torch.uint8, device="cuda")
        if rank == 0:
            import ctypes as C

            cbuf = (C.c_uint8 * 128)()
            capi.check(None, capi.load().ob_tp_unique_id(cbuf))
            buf.copy_(torch.tensor(list(cbuf), dtype=torch.uint8))
        dist.broadcast(buf, 0)
        return bytes(buf.cpu().tolist())

    uid = make_uid()

    ctx_len, K, W = args.context, args.steps, args.warmup
    b64 = args.batch64_steps
    margin = 2 * (K + W) + 96
    per_seq = ctx_len + margin
    model = orangu_b200.LlamaModel(be, cfg, tensors, max_seq_len=per_seq, max_batch_tokens=512,
                                   kv_pool_tokens=per_seq + (63 * (ctx_len + b64 + 64 + 16) if b64 else 0) + 64,
                                   tp_rank=rank, tp_size=world, tp_unique_id=uid, tp_presliced=world > 1)
    kv = model.new_kv_cache(per_seq)
    prompt = np.random.default_rng(11).integers(0, cfg["n_vocab"], ctx_len).astype(np.uint32)
    t_prefill = time.time()
    first = model.forward_maybe_sampling(kv, prompt, 0)
    t_prefill = time.time() - t_prefill

    sampler = ClockSampler(local_rank)
    # ---- value: device-resident loop -------------------------------------------------------------
    model.decode_loop([kv], [first], max(W, 3))
    barrier()
    sampler.start()
    launches0 = be.launch_count()
    out = model.decode_loop([kv], [int(first)], K)
    dev_ms = be.last_device_ms()
    launches = be.launch_count() - launches0
    barrier()
    dev_ms = max_over_ranks(dev_ms)
    value = K / (dev_ms * 1e-3)

    # ---- e2e: one host round trip per token --------------------------------------------------------
    tok = int(out[-1, 0])
    for _ in range(max(W, 3)):
        tok = model.decode_greedy(kv, tok)
    barrier()
    t0 = time.perf_counter()
    for _ in range(K):
        tok = model.decode_greedy(kv, tok)
    barrier()
    e2e_s = max_over_ranks(time.perf_counter() - t0)
    clocks = sampler.stop()
    T = model.max_batch_tokens
    h2d = ((T * 12 + 15) // 16) * 16 + T * 8  # the step's metadata block: token ids, positions, window lengths, page-table pointers
    e2e = {"value": K / e2e_s, "unit": UNIT, "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4, "ms_per_step": e2e_s / K * 1e3}

    # ---- roofline of the dominant kernel --------------------------------------------------------------
    peak, peak_kind = measured_peak_gbs()
    iters = 20
    step_bytes = algorithmic_bytes_per_token(cfg, len(kv)) // world
    # the fused decode kernels, each timed back to back over all layers (every launch streams its own layer's weights; on
    # several GPUs: this rank's slices); the gate/up kernel carries 43% of a token's bytes and is the one reported
    names = {1: "attn_q/k/v + RoPE + KV append", 2: "attn_output + residual", 3: "ffn_gate + ffn_up + SwiGLU + int8 output",
             4: "ffn_down + residual", 5: "output projection"}
    kernels = {}
    for v in (1, 2, 3, 4, 5):
        ms, nbytes, nl = model.profile_gemv(12, iters, v)
        us = max_over_ranks(ms * 1e3 / (iters * nl))
        kernels[names[v]] = {"avg_launch_us": us, "algorithmic_bytes_per_launch": nbytes // nl, "GB/s": nbytes / nl / us / 1e3,
                             "frac": nbytes / nl / us / 1e3 / peak, "launches_per_token": nl}
    dom = kernels[names[3]]
    kname = "stream_gemv_kernel<lanes per row pair 32, Q4_K> (" + names[3] + ")"
    per_launch_s, bytes_per_launch, timed = dom["avg_launch_us"] * 1e-6, dom["algorithmic_bytes_per_launch"], iters * cfg["n_layer"]
    achieved = bytes_per_launch / per_launch_s / 1e9
    # DRAM read + write bytes of one launch of the gate/up kernel of the 8B shape on one GPU, from the ncu capture of this kernel on
    # a two-layer model of the same shape (a capture cannot run inside a timed bench): dram__bytes_read.sum + dram__bytes_write.sum
    traffic = 66128896 + 896000 if world == 1 and (cfg["n_embd"], cfg["n_ff"]) == (4096, 14336) else None
    roofline = {"bound": "hbm", "kernel": kname, "achieved": achieved, "peak": peak, "peak_kind": peak_kind, "unit": "GB/s",
                "frac": achieved / peak, "traffic": traffic, "traffic_source": "profiles/decode_step_kernels_8b_ncu_full.md" if traffic else None,
                "launches_timed": timed, "avg_launch_us": per_launch_s * 1e6, "algorithmic_bytes_per_launch": bytes_per_launch,
                "step": {"algorithmic_bytes_per_token_per_gpu": step_bytes, "achieved": step_bytes / (dev_ms * 1e-3 / K) / 1e9,
                         "frac": step_bytes / (dev_ms * 1e-3 / K) / 1e9 / peak},
                "kernels": kernels}
    if world == 1:
        roofline["operator_gemv"] = operator_gemv_rooflines(be, peak)

    # ---- batch 64 extra ---------------------------------------------------------------------------------
    batch64 = None
    if b64:
        caches = [kv]
        for _ in range(63):
            c = model.new_kv_cache(ctx_len + b64 + 64)
            c.copy_prefix_from(kv, ctx_len)
            caches.append(c)
        kv.truncate(ctx_len)
        firsts = [int(first)] * 64
        model.decode_loop(caches, firsts, 3)
        barrier()
        out64 = model.decode_loop(caches, firsts, b64)
        ms64 = max_over_ranks(be.last_device_ms())
        batch64 = {"value": 64 * b64 / (ms64 * 1e-3), "unit": UNIT, "steps": b64, "ms_per_step": ms64 / b64, "sequences": 64,
                   "context": ctx_len, "kv": "63 sequences share the first one's prefilled pages by device copy (KvCache::copy_prefix_from)",
                   "algorithmic_bytes_per_step": algorithmic_bytes_per_token(cfg, 0) + 64 * (algorithmic_bytes_per_token(cfg, ctx_len) - algorithmic_bytes_per_token(cfg, 0))}
        batch64["hbm_frac_per_gpu"] = batch64["algorithmic_bytes_per_step"] / world / (ms64 / b64 * 1e-3) / 1e9 / peak
        batch64["parallelism"] = f"tp{world}"

    # ---- serving extra: eight request threads through the slot pool and the decode window (one GPU) ------------------------
    serving = None
    if b64 and world == 1:
        import threading

        from orangu_b200 import SlotPool

        for c in caches[1:]:
            c.close()  # their pages go back to the pool the slots draw from
        n_req, n_prompt, n_new = 8, 256, 33
        pool = SlotPool(model, n_slots=n_req, slot_capacity_tokens=n_prompt + n_new + 16, batch_wait_ms=0, prefill_batch=512, batch_decode=True)
        prompts = [np.random.default_rng(100 + i).integers(0, cfg["n_vocab"], n_prompt).astype(np.uint32) for i in range(n_req)]
        done_tokens, failures = [0] * n_req, []

        def request(i):
            try:
                with pool.try_acquire() as slot:
                    tok = slot.prefill(prompts[i])
                    for _ in range(n_new - 1):
                        tok = slot.decode(tok)
                        done_tokens[i] += 1
            except Exception as e:  # noqa: BLE001
                failures.append(repr(e)[:200])

        threads = [threading.Thread(target=request, args=(i,)) for i in range(n_req)]
        t0 = time.perf_counter()
        for t in threads:
            t.start()
        for t in threads:
            t.join()
        wall = time.perf_counter() - t0
        st = pool.stats()
        pool.close()
        serving = {"requests": n_req, "prompt_tokens": n_prompt, "new_tokens": n_new, "wall_s": wall,
                   "tok_s_generated": sum(done_tokens) / wall, "tok_s_prefill_and_decode": (n_req * n_prompt + sum(done_tokens)) / wall,
                   "decode_batches": st["batches"], "mean_decode_batch": st["batched_seqs"] / max(1, st["batches"]), "refused": st["refused"],
                   "failures": failures, "how": "one thread per request: ob_slot_acquire, ob_slot_prefill, ob_slot_decode per token through the default 4 ms "
                   "collection window, ob_slot_release; on-demand KV pages; host round trip per token"}

    # ---- CPU baseline (rank 0, single GPU runs only) --------------------------------------------------------
    cpu = None
    if rank == 0 and world == 1 and not args.no_cpu_baseline:
        v, cores, sample = cpu_decode_tokens_per_s(cfg, tensors, budget_s=15.0, max_tokens=400)
        cpu = {"value": v, "unit": UNIT, "cores": cores, "kind": "port", "sample": sample}

    # ---- 70B shape, tensor parallel (2, 4, 8 GPUs): batch 1 and batch 32 at context 8192 --------------------------------
    model70b = None
    if world > 1 and args.model == "8b" and not args.layers and os.environ.get("OB_BENCH_70B", "1") != "0":
        model.close()
        model = None
        try:
            model70b = run_70b(be, rank, world, make_uid(), barrier, max_over_ranks, peak)
        except Exception as e:  # the headline line must not depend on the extra
            model70b = {"error": f"{type(e).__name__}: {e}"[:300]}

    if rank == 0:
        line = {
            "metric": METRIC, "value": value, "unit": UNIT, "n_gpus": world, "steps": K, "warmup": max(W, 3), "ms_per_step": dev_ms / K,
            "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "int8", "data": "synthetic",
            "config": {"workload": f"{args.model}-shape Llama decoder, Q4_K_M (Q6_K output and attn_v), {cfg['n_layer']} layers, greedy decode at batch 1, "
                                   f"context {ctx_len} prefilled through the library, fp16 KV in 16-token pages",
                       "parallelism": f"tp{world}", "context": ctx_len, "batch": 1,
                       "l2": "inputs larger than L2: every step streams the whole quantized model (4.4 GB) through a 126 MB L2",
                       "attention": "windows above 1024 positions use the flash-decode kernel (not bit-exact: at this shape and context the logits differ from the "
                                    "CPU oracle by 0.10 max-abs at 2 layers and 0.17 at 4, above the 2e-2 bar, with identical greedy top-1; "
                                    "tests/test_gpu_model.py measures it); shorter windows use the exact-order kernels and are bit-identical",
                       "setup_s": {"synthetic_weights": round(t_build, 1), "prefill": round(t_prefill, 1)},
                       "launches_before_timed_region": int(launches0)},
            "clocks": clocks, "e2e": e2e, "gpu_launches": int(launches), "roofline": roofline, "cpu_baseline": cpu,
        }
        if batch64:
            line["batch64"] = batch64
        if serving:
            line["serving"] = serving
        if model70b:
            line["model70b"] = model70b
        print(json.dumps(line), flush=True)
    if model is not None:
        model.close()
    be.close()
    if world > 1:
        dist.destroy_process_group()


if __name__ == "__main__":
    main()
