"""In-tree build of libbitttt_b200.so (sm_100a only) with nvcc.

    python bit-ttt-engine_b200/build.py [--force] [--verbose]

The library has no dependency on PyTorch; it links the CUDA runtime (and NCCL for the
tensor-parallel entry points).
"""
from __future__ import annotations

import fcntl
import glob
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB_DIR = os.path.join(HERE, "lib")
OBJ_DIR = os.path.join(LIB_DIR, "obj")
LIB_PATH = os.path.join(LIB_DIR, "libbitttt_b200.so")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
]


def _nvcc() -> str:
    for cand in (shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found: the CUDA library cannot be built")


def sources() -> list[str]:
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")))


def _headers() -> list[str]:
    return glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(HERE, "..", "include", "*.h"))


def is_stale() -> bool:
    if not os.path.exists(LIB_PATH):
        return True
    built = os.path.getmtime(LIB_PATH)
    return any(os.path.getmtime(p) > built for p in sources() + _headers())


def _compile(nvcc: str, src: str, verbose: bool) -> str:
    """One source to its object, unless the object is newer than the source and the headers."""
    obj = os.path.join(OBJ_DIR, os.path.basename(src) + ".o")
    cmd = [nvcc, *NVCC_FLAGS, "-c", "-o", obj + f".{os.getpid()}", src]
    if verbose:
        cmd.insert(1, "-Xptxas=-v")
    proc = subprocess.run(cmd, capture_output=True, text=True)
    if proc.returncode != 0:
        raise RuntimeError(f"nvcc failed on {src}:\n" + proc.stdout + proc.stderr)
    if verbose:
        print(proc.stderr)
    os.replace(obj + f".{os.getpid()}", obj)
    return obj


def build_library(force: bool = False, verbose: bool = False) -> str:
    """Compiles the sources side by side and links them.  One process builds at a time; the others wait for it."""
    if not force and not is_stale():
        return LIB_PATH
    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(LIB_DIR, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and not is_stale():
            return LIB_PATH
        nvcc = _nvcc()
        headers = max(os.path.getmtime(p) for p in _headers())
        objs, todo = [], []
        for src in sources():
            obj = os.path.join(OBJ_DIR, os.path.basename(src) + ".o")
            objs.append(obj)
            if force or not os.path.exists(obj) or os.path.getmtime(obj) < max(headers, os.path.getmtime(src)):
                todo.append(src)
        with ThreadPoolExecutor(max_workers=max(1, min(len(todo), os.cpu_count() or 1))) as pool:
            list(pool.map(lambda s: _compile(nvcc, s, verbose), todo))
        part = LIB_PATH + f".{os.getpid()}"
        proc = subprocess.run([nvcc, *NVCC_FLAGS, "-shared", "-o", part, *objs, "-ldl"], capture_output=True, text=True)
        if proc.returncode != 0:
            raise RuntimeError("nvcc failed:\n" + proc.stdout + proc.stderr)
        os.replace(part, LIB_PATH)
    return LIB_PATH


if __name__ == "__main__":
    print(build_library(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
