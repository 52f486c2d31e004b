"""Compiles the backend in-tree: zeninfer_b200/lib/libzen_cuda.so (kernels + C-ABI, sm_100a only).

    python -m zeninfer_b200.build            # rebuild if sources are newer than the library
    python -m zeninfer_b200.build --force
"""
from __future__ import annotations

import fcntl
import os
import re
import shutil
import subprocess
import sys
import time

PKG = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG, "csrc")
LIB_DIR = os.path.join(PKG, "lib")
OBJ_DIR = os.path.join(LIB_DIR, "obj")
LIB = os.path.join(LIB_DIR, "libzen_cuda.so")
INCLUDE = os.path.join(os.path.dirname(PKG), "include")

NVCC_FLAGS = [
    "-std=c++17", "-O3", "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
]


def _sources() -> list[str]:
    return sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cu"))


def _inputs(source: str) -> set[str]:
    """A translation unit and everything of this repository it includes."""
    seen, todo = set(), [source]
    while todo:
        path = os.path.normpath(todo.pop())
        if path in seen or not os.path.exists(path):
            continue
        seen.add(path)
        with open(path) as f:
            todo += [os.path.join(os.path.dirname(path), name) for name in re.findall(r'^#include "([^"]+)"', f.read(), re.M)]
    return seen


def _stale(target: str, inputs) -> bool:
    return not os.path.exists(target) or os.path.getmtime(target) < max(os.path.getmtime(f) for f in inputs)


def build(force: bool = False, verbose: bool = False) -> str:
    """Returns the path of the built library; raises if nvcc is missing or compilation fails.  Translation units are compiled
    side by side, and only those whose sources changed; processes that ask for the library at the same time build it once."""
    inputs = {src: _inputs(src) for src in _sources()}
    everything = set().union(*inputs.values())
    if not force and not _stale(LIB, everything):
        return LIB
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(nvcc):
        if os.path.exists(LIB):
            return LIB  # a prebuilt library travelled with the tree
        raise RuntimeError("nvcc not found and no prebuilt libzen_cuda.so")
    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(OBJ_DIR, "lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and not _stale(LIB, everything):
            return LIB
        flags = ["-Xptxas=-v", *NVCC_FLAGS] if verbose else NVCC_FLAGS
        jobs, objects, began = [], [], time.time()
        for src, needs in inputs.items():
            obj = os.path.join(OBJ_DIR, os.path.basename(src)[:-3] + ".o")
            objects.append(obj)
            if force or _stale(obj, needs):
                cmd = [nvcc, *flags, "-I", INCLUDE, "-c", "-o", obj, src]
                jobs.append((cmd, subprocess.Popen(cmd)))
        codes = [(cmd, job.wait()) for cmd, job in jobs]
        for cmd, code in codes:
            if code:
                raise subprocess.CalledProcessError(code, cmd)
            os.utime(cmd[cmd.index("-o") + 1], (began, began))     # a source edited while it was compiled is newer than its object
        fresh = LIB + ".new"
        subprocess.run([nvcc, *NVCC_FLAGS, "-shared", "-o", fresh, *objects], check=True)
        os.utime(fresh, (began, began))
        os.replace(fresh, LIB)
    return LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
