"""Builds the CUDA library (kernels, C ABI, model drivers) for sm_100a.

Usage: python build.py [--target gpt2|decoder] [--force] [--verbose]
  gpt2     lib/libb200gpt2.so: everything
  decoder  lib/libb200decoder.so: the part of it that the layered decoders need, for a process that serves
           only such a model and finds nothing built
The libraries are written next to this file so that they travel with the source tree; they link only the
CUDA runtime (the driver API entry point they need is looked up at run time).
"""
from __future__ import annotations

import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB_DIR = os.path.join(HERE, "lib")
LIB_PATH = os.path.join(LIB_DIR, "libb200gpt2.so")
DECODER_LIB_PATH = os.path.join(LIB_DIR, "libb200decoder.so")

DECODER_SOURCES = [
    "api/ctx.cu",
    "kernels/rowwise.cu",
    "kernels/gemm_tf32.cu",
    "kernels/gemm_tf32_pair.cu",
    "kernels/decode.cu",
    "kernels/rmsnorm.cu",
    "kernels/gemm_fp32.cu",
    "kernels/gemm_decode.cu",
    "kernels/recurrent.cu",
    "kernels/experts.cu",
    "kernels/attention_latent.cu",
    "kernels/attention_cached.cu",
    "driver/decoder.cu",
]
SOURCES = DECODER_SOURCES + [
    "api/api.cu",
    "kernels/attention.cu",
    "kernels/attention_x3.cu",
    "kernels/attention_split.cu",
    "driver/gpt2.cu",
]
TARGETS = {"gpt2": (LIB_PATH, SOURCES), "decoder": (DECODER_LIB_PATH, DECODER_SOURCES)}

NVCC_FLAGS = [
    "-std=c++17", "-O3", "-lineinfo",
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=default",
    "--cudart", "shared",
]


def _sources_mtime() -> float:
    latest = 0.0
    for root, _, files in os.walk(CSRC):
        for f in files:
            latest = max(latest, os.path.getmtime(os.path.join(root, f)))
    latest = max(latest, os.path.getmtime(os.path.join(HERE, "..", "include", "b200gpt2.h")))
    return latest


def fresh(target: str = "gpt2") -> bool:
    """Whether the target's library is there and no older than the sources."""
    path = TARGETS[target][0]
    return os.path.exists(path) and os.path.getmtime(path) >= _sources_mtime()


def build(force: bool = False, verbose: bool = False, target: str = "gpt2") -> str:
    lib_path, sources = TARGETS[target]
    os.makedirs(LIB_DIR, exist_ok=True)
    if not force and fresh(target):
        return lib_path
    latest = _sources_mtime()
    obj_dir = os.path.join(HERE, "build")
    os.makedirs(obj_dir, exist_ok=True)
    objs, procs = [], []
    for src in sources:
        obj = os.path.join(obj_dir, src.replace("/", "_") + ".o")
        objs.append(obj)
        if not force and not verbose and os.path.exists(obj) and os.path.getmtime(obj) >= latest:
            continue  # compiled for the other target
        cmd = ["nvcc", *NVCC_FLAGS, "-c", os.path.join(CSRC, src), "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0 or verbose:
            sys.stderr.write(f"--- nvcc {src}\n{out}\n")
        failed |= p.returncode != 0
    if failed:
        raise RuntimeError(f"nvcc failed building {os.path.basename(lib_path)}")
    # linked beside its place and moved there, so that a process that finds the library finds all of it
    part = f"{lib_path}.{os.getpid()}.part"
    subprocess.check_call(["nvcc", "-gencode", "arch=compute_100a,code=sm_100a", "-shared", "--cudart", "shared", "-o", part, *objs])
    os.replace(part, lib_path)
    return lib_path


if __name__ == "__main__":
    which = sys.argv[sys.argv.index("--target") + 1] if "--target" in sys.argv else "gpt2"
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, target=which))
