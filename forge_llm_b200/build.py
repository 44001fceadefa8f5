"""Builds ``libforge_b200.so`` (the CUDA kernels and the C ABI) in-tree with nvcc for sm_100a.

    python -m forge_llm_b200.build [--force] [--verbose]
"""
from __future__ import annotations

import hashlib
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(CSRC, "build")
LIB = os.path.join(HERE, "libforge_b200.so")
STAMP = LIB + ".sha256"
SOURCES = ["pack.cu", "gemv_tc.cu", "gemv_batch.cu", "elementwise.cu", "attn_decode.cu", "attn_prefill_tc5.cu", "gemm_mma.cu", "gemm_tc5.cu",
           "tp_comm.cu", "gguf_reader.cu", "kquant_host.cu", "sampler.cu", "api_ops.cu", "model.cu",
           "checkpoint.cu", "gemm_dense.cu", "mla.cu", "mla_decode.cu", "attn_prefill_kv.cu", "attn_rows.cu", "moe.cu", "attn_pool.cu", "attn_talk.cu", "selective.cu", "recurrent.cu", "recurrent_chunk.cu", "stack_config.cu", "stack_model.cu"]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC,-fopenmp,-O3", "-Xptxas", "-v"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    return "nvcc"


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def build_library(force: bool = False, verbose: bool = False) -> str:
    os.makedirs(OBJ, exist_ok=True)
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    headers.append(os.path.join(HERE, "..", "include", "forge_b200.h"))
    nvcc = _nvcc()

    def compile_one(src: str):
        s = os.path.join(CSRC, src)
        o = os.path.join(OBJ, src.replace(".cu", ".o"))
        if force or _stale(o, [s] + headers):
            r = subprocess.run([nvcc, *NVCC_FLAGS, "-c", s, "-o", o], capture_output=True, text=True)
            if r.returncode != 0:
                raise RuntimeError(f"nvcc failed on {src}:\n{r.stdout}\n{r.stderr}")
            if verbose:
                print(f"== {src}\n{r.stderr}", file=sys.stderr)
            return o, True
        return o, False

    with ThreadPoolExecutor(max_workers=min(8, len(SOURCES))) as ex:
        results = list(ex.map(compile_one, SOURCES))
    objs = [o for o, _ in results]
    if force or any(c for _, c in results) or not os.path.exists(LIB):
        r = subprocess.run([nvcc, "--shared", "-o", LIB, *objs, "-Xcompiler", "-fopenmp", "-lgomp", "-ldl"],
                           capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    with open(STAMP, "w") as f:
        f.write(_digest() + "\n")
    return LIB


def _digest() -> str:
    """Content hash of everything the library is built from."""
    h = hashlib.sha256()
    files = sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cu", ".cuh", ".h")))
    for f in files + [os.path.join(HERE, "..", "include", "forge_b200.h"), os.path.abspath(__file__)]:
        h.update(os.path.basename(f).encode())
        with open(f, "rb") as fh:
            h.update(fh.read())
    return h.hexdigest()


def ensure_library() -> str:
    """Builds the library if it is missing or was built from other sources (by content, not by file times)."""
    try:
        with open(STAMP) as f:
            if f.read().strip() == _digest() and os.path.exists(LIB):
                return LIB
    except OSError:
        pass
    return build_library()


if __name__ == "__main__":
    print(build_library(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
