"""Builds libtlaloc_kernels.so (sm_100a) in-tree with nvcc.

    python -m tlaloc_b200.build [--force] [--verbose]

Each .cu under csrc/ is compiled to an object in build/ (in parallel) and the objects are linked into
tlaloc_b200/lib/libtlaloc_kernels.so, the name the reference's loaders look for
(triton/backend/pjrt_runtime.cc:139-164).  A target newer than every source is left alone, so machines
without nvcc (or without the sources' mtimes changing) just use the library that is there.

A process that serves one model needs only that model's kernels: `build(subset="latent")` compiles the sources listed in
SUBSETS (from the same objects) into a library of its own, unless the full library is there and current.
"""
from __future__ import annotations

import concurrent.futures
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB_DIR = os.path.join(HERE, "lib")
LIB = os.path.join(LIB_DIR, "libtlaloc_kernels.so")
SUBSETS = {"latent": ("runtime", "token_ops", "dense_gemm", "dense_gemm_tc", "latent_ops", "latent_attention", "latent_prefill"),
           "mixed": ("runtime", "token_ops", "dense_gemm", "dense_gemm_tc", "latent_ops", "latent_prefill", "mixer_ops", "grouped_attention",
                     "retention", "retention_chunks", "moe")}
INCLUDE = os.path.join(os.path.dirname(HERE), "include")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr", "-I", INCLUDE,
]


def library(subset: str | None = None) -> str:
    return LIB if subset is None else os.path.join(LIB_DIR, f"libtlaloc_{subset}.so")


def sources(subset: str | None = None) -> list[str]:
    names = sorted(f for f in os.listdir(CSRC) if f.endswith(".cu") and (subset is None or f[:-3] in SUBSETS[subset]))
    return [os.path.join(CSRC, f) for f in names]


def _deps(subset: str | None = None) -> list[str]:
    extra = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    return sources(subset) + extra + [os.path.join(INCLUDE, "tlaloc_b200.h")]


def up_to_date(subset: str | None = None) -> bool:
    lib = library(subset)
    if not os.path.exists(lib):
        return False
    t = os.path.getmtime(lib)
    return all(os.path.getmtime(d) <= t for d in _deps(subset))


def nvcc() -> str | None:
    return shutil.which("nvcc") or ("/usr/local/cuda/bin/nvcc" if os.path.exists("/usr/local/cuda/bin/nvcc") else None)


def build(force: bool = False, verbose: bool = False, subset: str | None = None, own: bool = False) -> str:
    """Path of an up-to-date library: the full one, or (subset given) one that holds at least the subset's kernels.  own: the
    subset's own library even where the full one would do."""
    lib = library(subset)
    if not force:
        for current in (subset,) if own else (None, subset):
            if up_to_date(current) and (current == subset or subset is not None):
                return library(current)
    cc = nvcc()
    if cc is None:
        for there in (lib, LIB):
            if os.path.exists(there):
                return there
        raise RuntimeError(f"nvcc not found and {os.path.basename(lib)} has not been built")
    os.makedirs(OBJ, exist_ok=True)
    os.makedirs(LIB_DIR, exist_ok=True)
    hdr_time = max(os.path.getmtime(d) for d in _deps(subset) if not d.endswith(".cu"))

    def compile_one(src: str) -> str:
        obj = os.path.join(OBJ, os.path.basename(src)[:-3] + ".o")
        if not force and os.path.exists(obj) and os.path.getmtime(obj) >= max(os.path.getmtime(src), hdr_time):
            return obj
        cmd = [cc, *NVCC_FLAGS, "-c", src, "-o", obj] + (["-Xptxas", "-v"] if verbose else [])
        r = subprocess.run(cmd, capture_output=True, text=True)
        if verbose or r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed on {src}")
        return obj

    with concurrent.futures.ThreadPoolExecutor(max_workers=8) as pool:
        objs = list(pool.map(compile_one, sources(subset)))
    r = subprocess.run([cc, "-shared", "-Xlinker", "--no-undefined", "-o", lib, *objs, "-gencode", "arch=compute_100a,code=sm_100a"],
                       capture_output=True, text=True)
    if r.returncode != 0:
        sys.stderr.write(r.stdout + r.stderr)
        raise RuntimeError("link failed")
    return lib


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
