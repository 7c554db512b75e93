"""Builds every CUDA source of this directory for sm_100a into one shared library next to the package.

Usage: ``python -m openrlhf_b200.csrc.build [--force] [--verbose] [--component NAME]``.
A component is a named subset of the sources linked into its own, smaller library: a process that only serves a model
(``component="serve_hybrid"``) can compile what that takes instead of the training kernels as well.
The library exports plain C symbols (see ``openrlhf_b200/ops/_lib.py`` for the prototypes) so that it has
no dependency on the PyTorch C++ headers and cross-compiles in seconds on a machine without a GPU.
"""
from __future__ import annotations

import hashlib
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
PKG = os.path.dirname(HERE)
LIB_NAME = "libopenrlhf_b200.so"
LIB_PATH = os.path.join(PKG, LIB_NAME)
OBJ_DIR = os.path.join(HERE, "build")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-lineinfo", "-std=c++17",
    "--use_fast_math",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]

# no fast-math: these kernels carry 32-bit recurrences, norms and logits and name their fast intrinsics one by one
PRECISE = {"hybrid_ops.cu", "ssd.cu", "ssd_chunk.cu", "attn_window.cu", "gemm_f32.cu"}

COMPONENTS = {
    "serve_hybrid": ["gemm_tcgen05.cu", "gemm2_tcgen05.cu", "sampling.cu", "host_runtime.cu",
                     "hybrid_ops.cu", "ssd.cu", "ssd_chunk.cu", "attn_window.cu", "attn_window_tc.cu",
                     "attn_decode.cu", "gemm_f32.cu"],
}


def component_path(component: str | None = None) -> str:
    return LIB_PATH if component is None else os.path.join(PKG, f"libopenrlhf_b200_{component}.so")


def _flags(src: str) -> list[str]:
    if os.path.basename(src) in PRECISE:
        return [f for f in NVCC_FLAGS if f != "--use_fast_math"]
    return NVCC_FLAGS


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    return "nvcc"


def sources(component: str | None = None) -> list[str]:
    names = [f for f in os.listdir(HERE) if f.endswith(".cu")] if component is None else COMPONENTS[component]
    return sorted(os.path.join(HERE, f) for f in names)


def _digest(path: str) -> str:
    h = hashlib.sha256()
    for dep in [path] + sorted(os.path.join(HERE, f) for f in os.listdir(HERE) if f.endswith((".cuh", ".h"))):
        with open(dep, "rb") as f:
            h.update(f.read())
    h.update(" ".join(_flags(path)).encode())
    return h.hexdigest()


def _compile_one(src: str, force: bool, verbose: bool) -> str:
    os.makedirs(OBJ_DIR, exist_ok=True)
    base = os.path.splitext(os.path.basename(src))[0]
    obj = os.path.join(OBJ_DIR, base + ".o")
    stamp = obj + ".sha"
    dig = _digest(src)
    if not force and os.path.exists(obj) and os.path.exists(stamp) and open(stamp).read() == dig:
        return obj
    cmd = [_nvcc(), *_flags(src), "-c", src, "-o", obj]
    if verbose:
        cmd.insert(1, "-Xptxas")
        cmd.insert(2, "-v")
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src}:\n{res.stdout}\n{res.stderr}")
    if verbose:
        sys.stderr.write(res.stderr)
    with open(stamp, "w") as f:
        f.write(dig)
    return obj


def build(force: bool = False, verbose: bool = False, component: str | None = None) -> str:
    srcs = sources(component)
    lib_path = component_path(component)
    with ThreadPoolExecutor(max_workers=min(8, len(srcs) or 1)) as ex:
        objs = list(ex.map(lambda s: _compile_one(s, force, verbose), srcs))
    newest = max(os.path.getmtime(o) for o in objs)
    if force or not os.path.exists(lib_path) or os.path.getmtime(lib_path) < newest:
        cmd = [_nvcc(), "-shared", "-o", lib_path, *objs, "-lcudart"]
        res = subprocess.run(cmd, capture_output=True, text=True)
        if res.returncode != 0:
            raise RuntimeError(f"link failed:\n{res.stdout}\n{res.stderr}")
    return lib_path


if __name__ == "__main__":
    path = build(force="--force" in sys.argv, verbose="--verbose" in sys.argv,
                 component=sys.argv[sys.argv.index("--component") + 1] if "--component" in sys.argv else None)
    print(path)
