"""Builds libjuno_b200.so (sm_100a only) in-tree with nvcc.

    python -m juno_b200.build            # incremental
    python -m juno_b200.build --force -v # rebuild, print ptxas resource usage
"""
from __future__ import annotations

import argparse
import concurrent.futures as cf
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB = os.path.join(HERE, "libjuno_b200.so")
SOURCES = ["context.cu", "gemv.cu", "qgemv.cu", "gemm.cu", "gemm_tc.cu", "attn.cu", "model.cu", "gguf_file.cu",
           "safetensors_file.cu", "registry.cu", "stack_loader.cu", "vosotar.cu", "desilorn.cu", "stack.cu", "stack_decode.cu", "gemv_rows.cu",
           "rowops.cu", "streams.cu", "gemm_rows.cu", "gemm_rows_tc.cu", "latent_attn.cu", "latent_attn_mma.cu", "flash_attn.cu",
           "grouped_attn.cu"]
ARCH = ["-gencode", "arch=compute_100a,code=sm_100a"]


def nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found")
    return exe


def _newest_header() -> float:
    t = 0.0
    for root in (CSRC, os.path.join(HERE, "..", "include")):
        for f in os.listdir(root):
            if f.endswith((".cuh", ".h", ".hpp")):
                t = max(t, os.path.getmtime(os.path.join(root, f)))
    return t


def _compile(src: str, verbose: bool) -> str:
    obj = os.path.join(OBJ, src.replace(".cu", ".o"))
    cmd = [nvcc(), *ARCH, "-O3", "-lineinfo", "-std=c++17", "--split-compile", "0", "-Xcompiler", "-fPIC,-O2", "-ccbin", "g++", "-c",
           os.path.join(CSRC, src), "-o", obj]
    if verbose:
        cmd += ["-Xptxas", "-v"]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src}:\n{r.stdout}\n{r.stderr}")
    if verbose:
        sys.stderr.write(r.stderr)
    return obj


def build(force: bool = False, verbose: bool = False) -> str:
    srcs = [s for s in SOURCES if os.path.exists(os.path.join(CSRC, s))]
    hdr_t = _newest_header()
    newest = max([hdr_t] + [os.path.getmtime(os.path.join(CSRC, s)) for s in srcs])
    if not force and os.path.exists(LIB) and os.path.getmtime(LIB) > newest:
        return LIB
    os.makedirs(OBJ, exist_ok=True)
    todo = []
    for s in srcs:
        obj = os.path.join(OBJ, s.replace(".cu", ".o"))
        if force or not os.path.exists(obj) or os.path.getmtime(obj) < max(os.path.getmtime(os.path.join(CSRC, s)), hdr_t):
            todo.append(s)
    if todo:
        with cf.ThreadPoolExecutor(max_workers=len(todo)) as ex:
            list(ex.map(lambda s: _compile(s, verbose), todo))
    objs = [os.path.join(OBJ, s.replace(".cu", ".o")) for s in srcs]
    if todo or not os.path.exists(LIB):
        cmd = [nvcc(), *ARCH, "-shared", "-o", LIB, *objs, "-ccbin", "g++", "-Xcompiler", "-fPIC", "-ldl"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    return LIB


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("-v", "--verbose", action="store_true")
    a = ap.parse_args()
    print(build(a.force, a.verbose))
