"""Compile the CUDA runtime in-tree for sm_100a (nvcc cross-compiles without a GPU)."""
from __future__ import annotations

import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "libfusekit_cuda.so")
SOURCES = ["fk_runtime.cu", "fk_layers.cu", "fk_blocks.cu"]        # compiled side by side, linked into one library
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-lineinfo", "-std=c++17",
         "-Xcompiler", "-fPIC", "-ccbin", "/usr/bin/g++"]


def _stale() -> bool:
    if not os.path.exists(OUT):
        return True
    t = os.path.getmtime(OUT)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if not f.endswith(".o")] + [os.path.join(HERE, "..", "include", "fusekit_cuda.h")]
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False) -> str:
    if force or _stale():
        objs = [os.path.join(CSRC, s[:-3] + ".o") for s in SOURCES]
        procs = [subprocess.Popen(["nvcc", *FLAGS, *(["-Xptxas", "-v"] if verbose else []), "-c", "-o", o, os.path.join(CSRC, s)])
                 for s, o in zip(SOURCES, objs)]
        codes = [p.wait() for p in procs]
        if any(codes):
            raise subprocess.CalledProcessError(next(c for c in codes if c), "nvcc")
        tmp = f"{OUT}.{os.getpid()}.tmp"                      # the finished library appears in one step
        subprocess.check_call(["nvcc", *FLAGS, "-shared", "-o", tmp, *objs, "-ldl"])
        os.replace(tmp, OUT)
    return OUT


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
