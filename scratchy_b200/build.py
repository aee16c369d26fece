"""Builds the C-ABI libraries in-tree with nvcc for sm_100a: ``libscratchy_cuda.so`` (quantized linears and the Llama
decode step) and ``libscratchy_models.so`` (the sequence-model kernels).

Usage: ``python -m scratchy_b200.build [--force] [--verbose]``.  nvcc cross-compiles
without a GPU; the resulting shared objects sit beside this file.  A program that serves one design of a source checkout
builds a library of that design's kernels only (`design_library`), so its first call compiles no more than it uses.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(CSRC, "build")
LIB = os.path.join(HERE, "libscratchy_cuda.so")
MODELS_LIB = os.path.join(HERE, "libscratchy_models.so")

SOURCES = ["context.cu", "abi.cu", "affine_b4.cu", "affine_b4_gemm.cu", "affine_b4_gemm_pair.cu", "fp8.cu", "fp8_gemm.cu", "fp8_gemm_pair.cu", "decode_ops.cu", "tp_comm.cu"]
MODELS_COMMON = ["context.cu", "dense_linear.cu", "dense_gemm.cu", "seq_ops.cu"]
# what the layers of a design run on
DESIGNS = {
    "Vumipel": ["latent_attention.cu", "latent_attention_mma.cu", "latent_prefill.cu", "mlstm.cu", "mlstm_chunk.cu"],
    "Vekurax": ["window_attention.cu", "window_attention_mma.cu", "window_prefill.cu", "lightning.cu", "lightning_chunk.cu"],
}
MODELS_SOURCES = MODELS_COMMON + [s for sources in DESIGNS.values() for s in sources]


def design_path(name: str) -> str:
    return os.path.join(HERE, f"libscratchy_models_{name.lower()}.so")


LIBRARIES = {LIB: SOURCES, MODELS_LIB: MODELS_SOURCES, **{design_path(n): MODELS_COMMON + sources for n, sources in DESIGNS.items()}}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "--use_fast_math=false",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


def _newer(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return False
    t = os.path.getmtime(target)
    return all(os.path.getmtime(d) <= t for d in deps)


def build(force: bool = False, verbose: bool = False) -> str:
    """Every library of the package."""
    for target in (LIB, MODELS_LIB):
        build_library(target, force, verbose)
    return LIB


def design_library(name: str) -> str:
    """The library to run a design from: the whole one where it is up to date, else one with the design's own sources."""
    if up_to_date(MODELS_LIB):
        return MODELS_LIB
    return build_library(design_path(name))


def headers() -> list[str]:
    found = []
    for folder in (CSRC, os.path.join(os.path.dirname(HERE), "include")):
        found += [os.path.join(folder, f) for f in os.listdir(folder) if f.endswith((".cuh", ".h"))]
    return found


def up_to_date(target: str) -> bool:
    return _newer(target, headers() + [os.path.join(CSRC, s) for s in LIBRARIES[target]])


def build_library(target: str, force: bool = False, verbose: bool = False) -> str:
    nvcc = _nvcc()
    os.makedirs(OBJ, exist_ok=True)
    sources, shared = LIBRARIES[target], headers()
    if not force and up_to_date(target):
        return target
    objs = []
    procs = []
    for src in sources:
        s = os.path.join(CSRC, src)
        o = os.path.join(OBJ, src.replace(".cu", ".o"))
        objs.append(o)
        if not force and _newer(o, [s] + shared):
            continue
        cmd = [nvcc, *[f for f in NVCC_FLAGS if f != "--use_fast_math=false"], "-c", s, "-o", o]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0:
            failed = True
            sys.stderr.write(f"--- nvcc failed on {src}\n{out}\n")
        elif verbose or "warning" in out:
            sys.stderr.write(f"--- {src}\n{out}\n")
    if failed:
        raise RuntimeError("nvcc failed")
    if force or procs or not _newer(target, objs):
        subprocess.check_call([nvcc, "-shared", "-o", target, *objs, "-gencode", "arch=compute_100a,code=sm_100a",
                               "-Xcompiler", "-fPIC"])
    return target


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
