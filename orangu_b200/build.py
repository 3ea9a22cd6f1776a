"""Builds the native libraries in-tree.

  orangu_b200/_lib/liborangu_b200.so   CUDA kernels + C ABI, sm_100a only (nvcc)
  orangu_b200/_lib/libob_synth.so      synthetic weight builder (host, g++)

Run as ``python -m orangu_b200.build``.  nvcc cross-compiles without a GPU.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIBDIR = os.path.join(HERE, "_lib")
OBJDIR = os.path.join(LIBDIR, "obj")
LIB = os.path.join(LIBDIR, "liborangu_b200.so")
SYNTH_LIB = os.path.join(LIBDIR, "libob_synth.so")

LAYERED_LIB = os.path.join(LIBDIR, "liborangu_b200_layered.so")  # the same library without the quantized kernels

CORE_SOURCES = ["api.cu", "model.cu", "tp.cu", "noalloc.cu", "gguf.cu", "sched.cu", "glue.cu", "linear.cu", "mixers.cu", "gqa.cu", "gqa_tc5.cu", "moe.cu", "recurrence.cu", "residual.cu", "layered.cu"]
QUANTIZED_SOURCES = ["formats.cu", "act_quant.cu", "gemv.cu", "attention.cu", "stream_gemv.cu", "layer_stream.cu", "gemm_mma.cu", "gemm_tc5.cu", "q5k.cu"]
CU_SOURCES = CORE_SOURCES + QUANTIZED_SOURCES
FMA_SOURCES = {"linear.cu", "mixers.cu", "gqa.cu", "gqa_tc5.cu", "moe.cu", "recurrence.cu", "residual.cu", "layered.cu"}  # no CPU arithmetic to reproduce: the compiler may fuse
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    # The reproduced arithmetic never fuses a*b+c; FMAs are written out where wanted.
    "-fmad=false",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


def _host_cxx() -> str:
    # the environment's CXX may be a g++ without libgomp
    return "/usr/bin/g++" if os.path.exists("/usr/bin/g++") else (shutil.which("g++") or "g++")


def _newer(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps if os.path.exists(d))


def _headers() -> list[str]:
    hs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    hs.append(os.path.join(os.path.dirname(HERE), "include", "orangu_b200.h"))
    return hs


def build_cuda(force: bool = False, verbose: bool = False, quantized: bool = True) -> str:
    """The whole library, or (quantized=False) what models given as a list of layers need."""
    sources, lib = (CU_SOURCES, LIB) if quantized else (CORE_SOURCES, LAYERED_LIB)
    os.makedirs(OBJDIR, exist_ok=True)
    nvcc = _nvcc()
    hdrs = _headers()
    jobs = []
    for src in sources:
        s = os.path.join(CSRC, src)
        o = os.path.join(OBJDIR, src.replace(".cu", ".o"))
        if force or _newer(o, [s] + hdrs):
            jobs.append((s, o))

    def compile_one(job):
        s, o = job
        flags = [f for f in NVCC_FLAGS if not (f == "-fmad=false" and os.path.basename(s) in FMA_SOURCES)]
        cmd = [nvcc, *flags, "-c", s, "-o", o]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed on {s}:\n{r.stdout}\n{r.stderr}")
        return r.stderr

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            for log in ex.map(compile_one, jobs):
                if verbose and log:
                    print(log, file=sys.stderr)
    objs = [os.path.join(OBJDIR, s.replace(".cu", ".o")) for s in sources]
    if force or jobs or _newer(lib, objs):
        cmd = [nvcc, "-shared", "-o", lib, *objs, "-gencode", "arch=compute_100a,code=sm_100a", "-Xcompiler", "-fPIC", "-ldl"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    return lib


def ensure_for(model_path: str) -> str:
    """The library a model needs, compiled if it is not there: the whole one when it is up to date or the model is quantized (a
    .gguf file), else the one without the quantized kernels.  Makes capi load it."""
    from . import capi

    sources = [os.path.join(CSRC, s) for s in CU_SOURCES] + _headers()
    whole = not _newer(LIB, sources)
    lib = LIB if whole else build_cuda(quantized=not os.path.isdir(model_path))
    capi.select(lib)
    return lib


def build_synth(force: bool = False) -> str:
    os.makedirs(LIBDIR, exist_ok=True)
    src = os.path.join(HERE, "synth", "synth.cpp")
    if force or _newer(SYNTH_LIB, [src]):
        # x86-64-v3, not -march=native: the library travels to other hosts
        cmd = [_host_cxx(), "-O3", "-march=x86-64-v3", "-fopenmp", "-fPIC", "-std=c++17", "-shared", "-o", SYNTH_LIB, src]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"g++ failed on synth.cpp:\n{r.stdout}\n{r.stderr}")
    return SYNTH_LIB


def build_all(force: bool = False, verbose: bool = False) -> None:
    build_cuda(force, verbose)
    build_synth(force)


if __name__ == "__main__":
    build_all(force="--force" in sys.argv, verbose="-v" in sys.argv)
    print(LIB)
    print(SYNTH_LIB)
