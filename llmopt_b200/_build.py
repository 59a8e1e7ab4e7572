"""Builds libllmopt_cuda.so in-tree with nvcc for sm_100a (no JIT cache, no torch)."""

from __future__ import annotations

import os
import subprocess
import sys
from typing import Optional

PACKAGE_DIR = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PACKAGE_DIR, "csrc")
LIBRARY = os.path.join(PACKAGE_DIR, "libllmopt_cuda.so")
OBJECTS = os.path.join(PACKAGE_DIR, "build")

# Kernel families that are enough to serve one kind of model: a host that needs no others can build
# and load libllmopt_cuda_<family>.so (the runtime registers only the names that were linked in).
_ATTENTION = ("runtime", "sampling", "dense_linear", "dense_gemm_tc", "sequence_glue", "row_attention", "experts")
FAMILIES = {
    "attention": _ATTENTION,  # decoders whose mixers all are attention
    "mixers": _ATTENTION + ("matrix_state",),
}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
]


def library_path(family: Optional[str] = None) -> str:
    return LIBRARY if family is None else os.path.join(PACKAGE_DIR, f"libllmopt_cuda_{family}.so")


def sources(family: Optional[str] = None) -> list[str]:
    names = sorted(name[:-3] for name in os.listdir(CSRC) if name.endswith(".cu"))
    return [os.path.join(CSRC, name + ".cu") for name in names if family is None or name in FAMILIES[family]]


def headers() -> list[str]:
    found = [os.path.join(CSRC, name) for name in os.listdir(CSRC) if name.endswith((".cuh", ".h"))]
    return found + [os.path.join(PACKAGE_DIR, "..", "include", "llmopt_cuda.h")]


def current(family: Optional[str] = None) -> bool:
    """Whether the library exists and is no older than its sources."""
    library = library_path(family)
    return os.path.exists(library) and not any(_newer(path, library) for path in sources(family) + headers())


def _newer(path: str, than: str) -> bool:
    return (not os.path.exists(than)) or os.path.getmtime(path) > os.path.getmtime(than)


def build(force: bool = False, verbose: bool = False, family: Optional[str] = None) -> str:
    """Compile changed translation units and link the shared library (of one family of kernels)."""
    nvcc = os.environ.get("NVCC", "nvcc")
    os.makedirs(OBJECTS, exist_ok=True)
    library = library_path(family)
    objects, jobs = [], []
    for source in sources(family):
        obj = os.path.join(OBJECTS, os.path.basename(source)[:-3] + ".o")
        objects.append(obj)
        stale = force or _newer(source, obj) or any(_newer(h, obj) for h in headers() if os.path.exists(h))
        if stale:
            command = [nvcc, *NVCC_FLAGS, "-c", source, "-o", obj]
            if verbose:
                command.insert(1, "-Xptxas=-v")
            jobs.append((source, subprocess.Popen(command, stdout=subprocess.PIPE, stderr=subprocess.STDOUT)))
    failed = False
    for source, job in jobs:
        output = job.communicate()[0].decode()
        if job.returncode != 0:
            failed = True
            sys.stderr.write(f"nvcc failed for {source}:\n{output}\n")
        elif verbose:
            sys.stderr.write(output)
    if failed:
        raise RuntimeError("libllmopt_cuda.so: compilation failed")
    if jobs or not os.path.exists(library) or any(_newer(obj, library) for obj in objects):
        subprocess.check_call(
            [nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "-shared", "-o", library, *objects, "-lcudart"]
        )
    return library


if __name__ == "__main__":
    chosen = [name for name in FAMILIES if f"--{name}" in sys.argv]
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, family=chosen[0] if chosen else None))
