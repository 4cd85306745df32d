"""In-tree build of the CUDA libraries for sm_100a with nvcc.

libllvq_b200.so serves archive-code (LLVQ) weights, libllvq_dense.so models with dense bf16 or f32 weights; a
process builds and loads only the one its model needs. The shared objects sit beside this file so that they
travel with the source tree; nothing is written to a per-user JIT cache.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libllvq_b200.so")
DENSE_LIB = os.path.join(HERE, "libllvq_dense.so")

SOURCES = {LIB: ["api.cu", "codebook.cpp", "tab_tables.cpp", "rotation.cpp", "archive.cpp"], DENSE_LIB: ["dense_api.cu"]}
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo", "--extended-lambda",
    "-Xcompiler", "-fPIC", "-shared", "-lcudart",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found; set NVCC or put it on PATH")


def _stale(lib: str) -> bool:
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC)]
    deps += [os.path.join(HERE, "..", "include", f) for f in ("llvq_b200.h", "llvq_dense.h")]
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False, lib: str = LIB) -> str:
    """Compile `lib` if it is missing or older than any source; return its path."""
    if not force and not _stale(lib):
        return lib
    part = f"{lib}.{os.getpid()}.part"  # moved into place when complete: another process never loads half a library
    cmd = [_nvcc(), *NVCC_FLAGS]
    if verbose:
        cmd += ["-Xptxas", "-v"]
    cmd += ["-o", part] + [os.path.join(CSRC, s) for s in SOURCES[lib]]
    res = subprocess.run(cmd, capture_output=True, text=True)
    if verbose or res.returncode:
        sys.stderr.write(res.stdout + res.stderr)
    if res.returncode:
        raise RuntimeError(f"nvcc failed building {os.path.basename(lib)}")
    os.replace(part, lib)
    return lib


if __name__ == "__main__":
    for target in SOURCES:
        print(build(force=True, verbose="-v" in sys.argv, lib=target))
