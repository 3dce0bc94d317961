"""Compile libtllm_b200.so in-tree with nvcc for sm_100a.

    python -m ternary_llm_b200.build [--force] [-v] [--timeline]

--timeline builds a second, diagnostic library, libtllm_b200_timeline.so, with
-DTLLM_TIMELINE: its GEMV kernels record time stamps of their phases (see
csrc/gemv_mma.cu) and it exports tllm_b200_timeline_read.  Point TLLM_B200_LIB at it to
load it instead of the regular library.

The library is a single shared object built from every .cu file under csrc/, each compiled to
an object of its own (build/, in parallel, only what changed).  nvcc cross-compiles without a
GPU, so this runs on a CPU-only build machine.
"""
from __future__ import annotations

import fcntl
import glob
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

PKG = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(PKG)
LIB = os.path.join(PKG, "libtllm_b200.so")
OBJ_DIR = os.path.join(ROOT, "build")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=default",
]


def sources():
    return sorted(glob.glob(os.path.join(PKG, "csrc", "*.cu")))


def headers():
    return glob.glob(os.path.join(PKG, "csrc", "*.cuh")) + glob.glob(os.path.join(ROOT, "include", "*.h"))


def _older(target: str, deps) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _stale() -> bool:
    return _older(LIB, sources() + headers())


def build(force: bool = False, verbose: bool = False, timeline: bool = False) -> str:
    out = os.path.join(PKG, "libtllm_b200_timeline.so") if timeline else LIB
    if not timeline and not force and not _stale():
        return LIB
    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(OBJ_DIR, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)         # two processes of a fresh checkout build it once
        if not timeline and not force and not _stale():
            return LIB
        flags = NVCC_FLAGS + (["-DTLLM_TIMELINE"] if timeline else []) + (["-Xptxas", "-v"] if verbose else []) + \
            ["-I" + os.path.join(ROOT, "include"), "-I" + os.path.join(PKG, "csrc")]
        suffix = ".timeline.o" if timeline else ".o"
        jobs = [(src, os.path.join(OBJ_DIR, os.path.splitext(os.path.basename(src))[0] + suffix)) for src in sources()]

        def compile_one(job):
            src, obj = job
            if force or verbose or _older(obj, [src] + headers()):
                part = obj + ".part"
                subprocess.check_call(["nvcc"] + flags + ["-c", "-o", part, src])
                os.replace(part, obj)

        with ThreadPoolExecutor(max(1, min(len(jobs), os.cpu_count() or 1))) as pool:
            list(pool.map(compile_one, jobs))
        part = out + ".part"
        subprocess.check_call(["nvcc"] + NVCC_FLAGS[:2] + ["-shared", "-o", part] + [obj for _, obj in jobs])
        os.replace(part, out)
    return out


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv, timeline="--timeline" in sys.argv))
