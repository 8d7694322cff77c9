"""Builds the sm_100a kernel library in-tree with nvcc.

Every ``csrc/*.cu`` file is compiled to an object (in parallel, only when its sources changed) and
linked into ``b200fw/_lib/libb200fw.so``.  The library exports plain C symbols taking raw device
pointers and a stream, so it needs neither the torch headers nor libcuda at link time and compiles in
seconds; :mod:`b200fw._native` binds it with ctypes.
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parent.parent
CSRC = ROOT / "csrc"
LIB_DIR = Path(__file__).resolve().parent / "_lib"
LIB_PATH = LIB_DIR / "libb200fw.so"
OBJ_DIR = LIB_DIR / "obj"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "--expt-relaxed-constexpr",
    "-Xcompiler", "-fPIC",
    "-Xcompiler", "-fvisibility=hidden",
]


def _nvcc() -> str:
    cand = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(cand):
        raise RuntimeError("nvcc not found; cannot build the b200fw kernel library")
    return cand


def _digest(paths) -> str:
    h = hashlib.sha256()
    h.update(" ".join(NVCC_FLAGS).encode())
    for p in sorted(paths):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    return h.hexdigest()


def sources():
    return sorted(CSRC.glob("*.cu"))


def partial_path(only) -> Path:
    return LIB_DIR / ("libb200fw_" + "_".join(sorted(only)) + ".so")


def build(verbose: bool = False, force: bool = False, only=None) -> Path:
    """Compile (if stale) and return the path of the shared library.  ``only``: stems of the sources to put into a smaller
    library of their own (for a process that needs few kernels and should not wait for the others)."""
    chosen = [p for p in sources() if only is None or p.stem in only]
    if only is not None and len(chosen) != len(set(only)):
        raise ValueError(f"unknown sources: {sorted(set(only) - {p.stem for p in chosen})}")
    lib_path = LIB_PATH if only is None else partial_path(only)
    OBJ_DIR.mkdir(parents=True, exist_ok=True)
    headers = sorted(list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h")))
    nvcc = _nvcc()
    jobs = []
    for src in chosen:
        obj = OBJ_DIR / (src.stem + ".o")
        stamp = OBJ_DIR / (src.stem + ".sha")
        dig = _digest([src] + headers)
        if force or not obj.exists() or not stamp.exists() or stamp.read_text() != dig:
            jobs.append((src, obj, stamp, dig))

    def compile_one(job):
        src, obj, stamp, dig = job
        cmd = [nvcc, *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            sys.stderr.write(r.stderr)
        stamp.write_text(dig)
        return src.name

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            list(ex.map(compile_one, jobs))
    objs = [OBJ_DIR / (s.stem + ".o") for s in chosen]
    if jobs or not lib_path.exists():
        cmd = [nvcc, "-shared", "-o", str(lib_path), *map(str, objs), "-cudart", "static"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    return lib_path


if __name__ == "__main__":
    p = build(verbose="-v" in sys.argv, force="-f" in sys.argv)
    print(p)
