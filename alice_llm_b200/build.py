"""Builds libalice_cuda.so (the C-ABI library of include/alice_cuda.h) for sm_100a with nvcc.

The same command line is what a Rust `build.rs` of the reference crate would run; it needs no
GPU (nvcc cross-compiles). Output: alice_llm_b200/libalice_cuda.so, kept in-tree.
"""
from __future__ import annotations

import os
from concurrent.futures import ThreadPoolExecutor
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libalice_cuda.so")
# What a layer-stack model needs, as a library of its own; the whole library is these and the quantized-matvec path.
LIB_STACK = os.path.join(HERE, "libalice_stack.so")
STACK_SOURCES = ["engine.cu", "tp.cu", "step.cu", "model_api.cu", "stack_model.cu", "stack_ops.cu", "dense_rows.cu", "dense_gemm.cu", "delta.cu",
                 "latent.cu", "latent_decode.cu", "latent_prefill.cu", "grouped.cu", "grouped_decode.cu", "grouped_prefill.cu"]
SOURCES = STACK_SOURCES + ["abi.cu", "gemv_launch.cu", "q8k.cu", "dequant.cu", "ternarize.cu", "glue.cu", "model.cu"]
# never --use_fast_math: dequantization and the Q8_K quantizer must round like the reference
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-fno-strict-aliasing"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    raise RuntimeError("nvcc not found")


def stale(lib: str) -> bool:
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if not f.endswith(".o")] + [os.path.join(HERE, "..", "include", "alice_cuda.h")]
    return any(os.path.getmtime(d) > t for d in deps)


def _object_stale(obj: str, src: str) -> bool:
    """Objects of unchanged sources are kept; any header change rebuilds them all."""
    if not os.path.exists(obj):
        return True
    t = os.path.getmtime(obj)
    deps = [src] + [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cuh")] + [os.path.join(HERE, "..", "include", "alice_cuda.h")]
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False, part: str = "all") -> str:
    """part "all": the complete library; "stack": only what layer-stack models need."""
    lib, sources = (LIB_STACK, STACK_SOURCES) if part == "stack" else (LIB, SOURCES)
    if not force and not stale(lib):
        return lib

    def compile_one(src):
        path, obj = os.path.join(CSRC, src), os.path.join(CSRC, src.replace(".cu", ".o"))
        if not force and not _object_stale(obj, path):
            return obj
        cmd = [_nvcc(), *NVCC_FLAGS, "-c", path, "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        subprocess.check_call(cmd)
        return obj

    # the translation units are independent: compile them side by side
    with ThreadPoolExecutor(max_workers=min(len(sources), os.cpu_count() or 1)) as pool:
        objs = list(pool.map(compile_one, sources))
    subprocess.check_call([_nvcc(), "-shared", "-o", lib, *objs, "-lcudart", "-ldl"])
    return lib


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv, part="stack" if "--stack" in sys.argv else "all"))
