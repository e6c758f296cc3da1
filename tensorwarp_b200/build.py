"""Ahead-of-time build of the kernel libraries for sm_100a with nvcc.

Two libraries, compiled in-tree: ``libtwmarlin.so`` (the 4-bit GEMM family and its decode step) and
``libtwmdense.so`` (decoder models with 16-bit or 32-bit weights).  There is no JIT of kernels at
run time; a model that needs a library which is not there yet has it compiled once, on first use.
nvcc cross-compiles without a GPU.
"""
from __future__ import annotations

import fcntl
import os
import subprocess
import sys
import tempfile

PKG = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG, "csrc")
INCLUDE = os.path.join(PKG, "..", "include")
LIB = os.path.join(PKG, "libtwmarlin.so")

# library -> (source, output)
TARGETS = {
    "marlin": ("twmarlin.cu", LIB),
    "dense": ("twm_dense.cu", os.path.join(PKG, "libtwmdense.so")),
}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-lineinfo", "-std=c++17",
    "-Xcompiler", "-fPIC", "-shared",
]


def _sources():
    out = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cu", ".cuh", ".hpp"))]
    out += [os.path.join(INCLUDE, f) for f in os.listdir(INCLUDE) if f.endswith(".h")]
    return sorted(out)


def _deps(target: str):
    """Every header, and the target's own .cu file."""
    own = TARGETS[target][0]
    return [s for s in _sources() if not s.endswith(".cu") or os.path.basename(s) == own]


def needs_build(target: str = "marlin") -> bool:
    lib = TARGETS[target][1]
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    return any(os.path.getmtime(s) > t for s in _deps(target))


def _nvcc() -> str:
    home = os.environ.get("CUDA_HOME", "/usr/local/cuda")
    path = os.path.join(home, "bin", "nvcc")
    return path if os.path.exists(path) else "nvcc"


def _compile(target: str, verbose: bool) -> None:
    src, lib = TARGETS[target]
    fd, part = tempfile.mkstemp(dir=PKG, prefix=".build-", suffix=".so")      # moved into place when complete
    os.close(fd)
    try:
        cmd = [_nvcc()] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + [os.path.join(CSRC, src), "-o", part]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if verbose:
            sys.stderr.write(r.stdout + r.stderr)
        if r.returncode != 0:
            raise RuntimeError("nvcc failed:\n" + r.stdout + r.stderr)
        os.chmod(part, 0o755)
        os.replace(part, lib)
    finally:
        if os.path.exists(part):
            os.unlink(part)


def build_library(target: str, force: bool = False, verbose: bool = False) -> str:
    """Compile one library if it is missing or older than its sources; one process at a time."""
    lib = TARGETS[target][1]
    if not force and not needs_build(target):
        return lib
    with open(os.path.join(PKG, f".build-{target}.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if force or needs_build(target):
            _compile(target, verbose)
    return lib


def build(force: bool = False, verbose: bool = False) -> str:
    """Compile every library of the package; returns the path of ``libtwmarlin.so``."""
    for target in TARGETS:
        build_library(target, force, verbose)
    return LIB


if __name__ == "__main__":
    build(force=True, verbose="-v" in sys.argv)
    for _, path in TARGETS.values():
        print(path)
