"""Builds the sm_100a kernel library in-tree with nvcc.

Every ``csrc/*.cu`` is compiled to an object (in parallel) and linked into
``areal_b200/ops/libab2_kernels.so``. The library exposes a plain C ABI that
``areal_b200.ops.lib`` loads with ctypes, so no PyTorch headers are involved and a full
rebuild takes seconds. nvcc cross-compiles without a GPU.

Usage: ``python -m areal_b200.ops.build [--force] [--verbose]``
"""
from __future__ import annotations

import argparse
import concurrent.futures as cf
import hashlib
import os
import shutil
import subprocess
import sys
from pathlib import Path

HERE = Path(__file__).resolve().parent
CSRC = HERE / "csrc"
BUILD = HERE / "build"
LIB = HERE / "libab2_kernels.so"
# the kernels that serve any mixer stack; with those of a design's own mixers, linked alone, they are what a fresh checkout
# compiles before its first trace
STEP_SOURCES = ("runtime", "gemm", "gemm2sm", "infer", "mixer_ops")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xptxas", "-v",
]


def _nvcc() -> str:
    cand = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(cand):
        raise RuntimeError("nvcc not found; the kernel library needs the CUDA toolkit")
    return cand


def _digest(paths) -> str:
    h = hashlib.sha256()
    for p in sorted(paths):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    h.update(" ".join(NVCC_FLAGS).encode())
    return h.hexdigest()


def sources(names=None):
    return sorted(p for p in CSRC.glob("*.cu") if names is None or p.stem in names)


def _headers() -> list:
    return list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h"))


def is_current(lib: Path = LIB, names=None) -> bool:
    stamp = BUILD / ("stamp" if lib == LIB else "stamp-" + lib.stem)
    if not lib.exists() or not stamp.exists():
        return False
    return stamp.read_text().strip() == _digest(sources(names) + _headers())


def build_step_library(design: str, own: tuple) -> Path:
    """The library a mixer stack is served from: the whole one when it is up to date, else the sources of every stack and the
    design's ``own``."""
    return LIB if is_current() else build(lib=HERE / f"libab2_step_{design}.so", names=STEP_SOURCES + own)


def build(force: bool = False, verbose: bool = False, lib: Path = LIB, names=None) -> Path:
    """Compiles and links the library if sources changed. Returns the library path. ``names``: the sources of a
    library that holds a subset of the kernels."""
    if not force and is_current(lib, names):
        return lib
    BUILD.mkdir(exist_ok=True)
    nvcc = _nvcc()
    srcs = sources(names)
    logs = {}

    def compile_one(src: Path):
        obj = BUILD / (src.stem + ".o")
        cmd = [nvcc, *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        return src, obj, r

    with cf.ThreadPoolExecutor(max_workers=min(8, len(srcs))) as ex:
        results = list(ex.map(compile_one, srcs))
    objs = []
    for src, obj, r in results:
        logs[src.name] = r.stderr
        if r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError(f"nvcc failed on {src.name}")
        if verbose:
            sys.stderr.write(f"== {src.name}\n{r.stderr}\n")
        objs.append(str(obj))
    (BUILD / "ptxas.log").write_text("\n".join(f"== {k}\n{v}" for k, v in logs.items()))
    part = lib.with_suffix(".part.so")
    link = [nvcc, "-shared", "-o", str(part), *objs, "-lcudart"]
    r = subprocess.run(link, capture_output=True, text=True)
    if r.returncode != 0:
        sys.stderr.write(r.stdout + r.stderr)
        raise RuntimeError("link failed")
    os.replace(part, lib)
    (BUILD / ("stamp" if lib == LIB else "stamp-" + lib.stem)).write_text(_digest(srcs + _headers()))
    return lib


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    a = ap.parse_args()
    print(build(force=a.force, verbose=a.verbose))
