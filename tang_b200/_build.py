"""Ahead-of-time build (nvcc, sm_100a only) next to this file: libtangq.so with every source, or -- for a process that
only needs one model family in a fresh checkout -- a smaller library with that family's sources behind the same ABI."""
from __future__ import annotations

import glob
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libtangq.so")
OBJ = os.path.join(HERE, "build")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
]

# sources of the partial libraries (name -> csrc/*.cu stems)
COMPONENTS = {
    "dense": ["api_core", "graph", "ops", "sampler", "dense", "rowops", "expert_route", "diff_attention",
              "window_attention", "gla", "gla_chunk", "lightning", "stream_mix", "latent_attention", "short_conv", "min_gru", "expert_ff",
              "tofazen", "numuzen", "dotanex", "sakinex"],
}


def sources(component: str | None = None) -> list[str]:
    if component is None:
        return sorted(glob.glob(os.path.join(CSRC, "*.cu")))
    return [os.path.join(CSRC, s + ".cu") for s in COMPONENTS[component]]


def library_path(component: str | None = None) -> str:
    return LIB if component is None else os.path.join(HERE, f"libtangq_{component}.so")


def _headers() -> list[str]:
    return glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h")) + [
        os.path.join(os.path.dirname(HERE), "include", "tangq.h")]


def _newer(deps, target: str) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def stale(component: str | None = None) -> bool:
    return _newer(sources(component) + _headers(), library_path(component))


def build_library(force: bool = False, verbose: bool = False, component: str | None = None) -> str:
    """Compiles the sources (in parallel, objects kept in build/) and links the library.  Needs nvcc, not a GPU."""
    lib = library_path(component)
    if not force and not stale(component):
        return lib
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    os.makedirs(OBJ, exist_ok=True)
    tag = f".{os.getpid()}"

    def compile_one(src: str) -> str:
        obj = os.path.join(OBJ, os.path.basename(src)[:-3] + ".o")
        if force or _newer([src, *_headers()], obj):
            cmd = [nvcc, *NVCC_FLAGS, *(["-Xptxas", "-v"] if verbose else []), "-c", "-o", obj + tag, src]
            subprocess.run(cmd, check=True, stdout=sys.stderr)
            os.replace(obj + tag, obj)
        return obj

    with ThreadPoolExecutor(max_workers=os.cpu_count() or 1) as pool:
        objs = list(pool.map(compile_one, sources(component)))
    subprocess.run([nvcc, *NVCC_FLAGS[:2], "-shared", "-ldl", "-o", lib + tag, *objs], check=True, stdout=sys.stderr)
    os.replace(lib + tag, lib)
    return lib


def ensure(component: str) -> str:
    """Path of a library that has `component`: the full one when it is up to date, else the partial one, built if needed."""
    if not stale():
        return LIB
    return build_library(component=component)


if __name__ == "__main__":
    print(build_library(force=True, verbose=True))
