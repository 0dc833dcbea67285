"""Builds libctox_b200.so in-tree with nvcc for sm_100a (cross-compiles without a GPU).

Every source becomes an object under build/ (only stale ones are compiled, several at a time); the
library is linked from them.
"""
from __future__ import annotations

import glob
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

PKG_DIR = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG_DIR, "csrc")
OBJ_DIR = os.path.join(PKG_DIR, "build")
LIB_PATH = os.path.join(PKG_DIR, "libctox_b200.so")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-lineinfo", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "-cudart", "static",
]


def sources() -> list[str]:
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")))


def _headers() -> list[str]:
    return glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(PKG_DIR, "..", "include", "*.h"))


def _older(target: str, deps) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def is_stale() -> bool:
    return _older(LIB_PATH, sources() + _headers())


def build(force: bool = False, verbose: bool = False) -> str:
    if not force and not is_stale():
        return LIB_PATH
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    os.makedirs(OBJ_DIR, exist_ok=True)
    common = _headers() + [os.path.abspath(__file__)]

    def compile_one(src: str) -> str:
        obj = os.path.join(OBJ_DIR, os.path.splitext(os.path.basename(src))[0] + ".o")
        if force or _older(obj, [src] + common):
            subprocess.check_call([nvcc] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) +
                                  ["-c", src, "-o", obj])
        return obj

    # largest source first: it decides when the parallel part ends
    srcs = sorted(sources(), key=os.path.getsize, reverse=True)
    with ThreadPoolExecutor(max_workers=max(1, os.cpu_count() or 1)) as pool:
        objs = list(pool.map(compile_one, srcs))
    # link beside the target and rename: another process never loads a half-written library
    tmp = f"{LIB_PATH}.{os.getpid()}.tmp"
    subprocess.check_call([nvcc] + NVCC_FLAGS + ["-shared", "-o", tmp] + sorted(objs))
    os.replace(tmp, LIB_PATH)
    return LIB_PATH


if __name__ == "__main__":
    build(force=True, verbose="-v" in sys.argv)
    print(LIB_PATH)
