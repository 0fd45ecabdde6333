"""Builds libdoppler_b200.so (CUDA, sm_100a) in-tree with nvcc.

Usage: python -m doppler_b200.build [--force] [--verbose]
"""
from __future__ import annotations

import concurrent.futures as cf
import fcntl
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "_build")
LIB = os.path.join(HERE, "libdoppler_b200.so")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", shutil.which("nvcc")):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


def _host_cxx() -> list[str]:
    # the distribution g++; a wrapper g++ earlier on PATH may lack pieces
    return ["-ccbin", "/usr/bin/g++"] if os.path.exists("/usr/bin/g++") else []


def sources() -> list[str]:
    return sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cu"))


def _deps_mtime() -> float:
    hdrs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    hdrs.append(os.path.join(HERE, "..", "include", "doppler_b200.h"))
    return max(os.path.getmtime(h) for h in hdrs)


def build(force: bool = False, verbose: bool = False) -> str:
    """Compile what is missing or older than its sources; one process at a time, outputs appear whole."""
    os.makedirs(OBJ, exist_ok=True)
    with open(os.path.join(OBJ, "lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build(force, verbose)


def _compile(cmd: list[str], out: str) -> subprocess.CompletedProcess:
    part = f"{out}.part{os.path.splitext(out)[1]}"
    res = subprocess.run([part if c == out else c for c in cmd], capture_output=True, text=True)
    if res.returncode == 0:
        os.replace(part, out)
    return res


def _build(force: bool, verbose: bool) -> str:
    nvcc, dep_t = _nvcc(), _deps_mtime()
    jobs = []
    for src in sources():
        obj = os.path.join(OBJ, os.path.basename(src)[:-3] + ".o")
        if force or not os.path.exists(obj) or os.path.getmtime(obj) < max(os.path.getmtime(src), dep_t):
            cmd = [nvcc, *_host_cxx(), *NVCC_FLAGS, "-c", src, "-o", obj]
            if verbose:
                cmd.insert(1, "-Xptxas=-v")
            jobs.append(cmd)
    if jobs:
        with cf.ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            for cmd, res in zip(jobs, ex.map(lambda c: _compile(c, c[-1]), jobs)):
                if verbose and res.stderr:
                    print(res.stderr, file=sys.stderr)
                if res.returncode != 0:
                    raise RuntimeError("nvcc failed: %s\n%s\n%s" % (" ".join(cmd), res.stdout, res.stderr))
    objs = [os.path.join(OBJ, os.path.basename(s)[:-3] + ".o") for s in sources()]
    if jobs or not os.path.exists(LIB):
        cmd = [nvcc, *_host_cxx(), "-shared", "-o", LIB, *objs, "-ldl", "-lpthread"]
        res = _compile(cmd, LIB)
        if res.returncode != 0:
            raise RuntimeError("link failed: %s\n%s" % (" ".join(cmd), res.stderr))
    return LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
