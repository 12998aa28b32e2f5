"""Builds libwick_cuda.so in-tree with nvcc for sm_100a.

`--fmad=false` is part of the numerics contract, not a tuning knob: the CPU path the
kernels must match bit for bit never contracts a*b+c, and the kernels call fmaf
explicitly where the reference uses a fused NEON instruction.
"""
from __future__ import annotations

import fcntl
import os
import re
import shutil
import subprocess
import sys
from typing import List

_HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(_HERE, "csrc")
LIB_PATH = os.path.join(_HERE, "libwick_cuda.so")
SOURCES = ["kernels_basic.cu", "kernels_gemv.cu", "kernels_attn.cu", "kernels_q6k.cu", "kernels_batch.cu", "kernels_sample.cu", "tp_comm.cu", "decode_mega.cu", "gemm_tc.cu", "argmax_noalloc.cu",
           "kernels_hyper.cu", "kernels_residual.cu", "kernels_dense.cu", "kernels_route.cu", "gemm_bf16.cu", "kernels_mixattn.cu", "attn_mix_tc.cu", "kernels_delta.cu", "delta_chunk.cu", "kernels_latent.cu", "attn_latent_step.cu", "attn_latent_tc.cu", "kernels_memory.cu", "memory_tc.cu", "hybrid_ops.cu", "hybrid_load.cu", "hybrid.cu", "wick_cuda.cu"]

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo", "--fmad=false",
    "-Xcompiler", "-fPIC,-Wall",
]


# sources of many large kernels: their code generation runs on several threads
SPLIT = {"delta_chunk.cu": ["--split-compile=0"]}


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


_INCLUDE = re.compile(r'^\s*#include "([^"]+)"', re.M)


def _newest(path: str, seen: set) -> float:
    """Newest modification time of a source and of what it includes from this repository."""
    seen.add(path)
    t = os.path.getmtime(path)
    with open(path) as f:
        text = f.read()
    for name in _INCLUDE.findall(text):
        inc = os.path.normpath(os.path.join(os.path.dirname(path), name))
        if inc not in seen and os.path.exists(inc):
            t = max(t, _newest(inc, seen))
    return t


def _read(path: str) -> str:
    try:
        with open(path) as f:
            return f.read()
    except OSError:
        return ""


def _inputs() -> dict:
    """Per source: newest modification time of what its object depends on."""
    return {f: _newest(os.path.join(CSRC, f), set()) for f in SOURCES}


def build(force: bool = False, verbose: bool = False, extra: List[str] | None = None) -> str:
    """Compiles what is out of date and links; safe to call from several processes at once."""
    srcs = _inputs()
    newest = max(srcs.values())
    newest = max(newest, os.path.getmtime(__file__))
    if not force and os.path.exists(LIB_PATH) and os.path.getmtime(LIB_PATH) >= newest:
        return LIB_PATH
    objdir = os.path.join(_HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    with open(os.path.join(objdir, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and os.path.exists(LIB_PATH) and os.path.getmtime(LIB_PATH) >= newest:
            return LIB_PATH  # another process has just done it
        return _compile(objdir, srcs, force or bool(extra), verbose, extra or [])


def _compile(objdir: str, srcs: dict, force: bool, verbose: bool, extra: List[str]) -> str:
    nvcc = _nvcc()
    env = dict(os.environ)
    # the environment may export CC/CXX pointing at a non-system compiler; nvcc wants the system g++
    ccbin = "/usr/bin/g++" if os.path.exists("/usr/bin/g++") else "g++"
    objs = []
    procs = []
    for src in SOURCES:
        obj = os.path.join(objdir, src.replace(".cu", ".o"))
        objs.append(obj)
        flags = " ".join([*NVCC_FLAGS, *SPLIT.get(src, []), *extra])
        if not force and os.path.exists(obj) and os.path.getmtime(obj) >= srcs[src] and _read(obj + ".flags") == flags:
            continue
        part = f"{obj}.{os.getpid()}.part.o"
        cmd = [nvcc, "-ccbin", ccbin, *NVCC_FLAGS, *SPLIT.get(src, []), *extra, "-c", os.path.join(CSRC, src), "-o", part]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        procs.append((cmd, part, obj, flags, subprocess.Popen(cmd, env=env, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = None
    for cmd, part, obj, flags, p in procs:
        out, _ = p.communicate()
        if verbose or p.returncode:
            sys.stderr.write(out)
        if p.returncode:
            failed = failed or cmd
        else:
            os.replace(part, obj)
            with open(obj + ".flags", "w") as f:
                f.write(flags)
    if failed:
        raise RuntimeError("nvcc failed: " + " ".join(failed))
    part = f"{LIB_PATH}.{os.getpid()}.part"
    link = [nvcc, "-ccbin", ccbin, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", part, *objs]
    subprocess.check_call(link, env=env)
    os.replace(part, LIB_PATH)
    return LIB_PATH


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
