"""Builds the sm_100a kernel library in-tree with nvcc (``smcsd_b200/ops/libsmcsd_b200.so``).

The library exposes plain ``extern "C"`` launchers that take raw device pointers and a
stream, so it has no build-time dependency on PyTorch and compiles in seconds.
Run ``python -m smcsd_b200.ops.build`` (add ``-v`` for ptxas register / spill output).
"""
from __future__ import annotations

import hashlib
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "libsmcsd_b200.so")
OBJ_DIR = os.path.join(HERE, "build")
ARCH = ["-gencode", "arch=compute_100a,code=sm_100a"]
# Sources whose fp32 arithmetic serves 32-bit runs: compiled with IEEE division, square root and exponentials.
PRECISE = {"chunk_attention.cu", "conv_act.cu", "conv_heads.cu", "gated_chunk.cu", "gated_memory.cu", "gemm_f32.cu", "hyper.cu", "latent_attention.cu", "memory_scan.cu",
           "memory_step.cu",            "moe.cu", "post_norm.cu", "side_norm.cu"}


def sources():
    return sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cu"))


def _digest() -> str:
    h = hashlib.sha256()
    for f in sorted(os.listdir(CSRC)):
        with open(os.path.join(CSRC, f), "rb") as fh:
            h.update(f.encode())
            h.update(fh.read())
    return h.hexdigest()


def nvcc_path() -> str:
    for c in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if c and (os.path.isabs(c) and os.path.exists(c) or not os.path.isabs(c)):
            return c
    return "nvcc"


def build(verbose: bool = False, force: bool = False) -> str:
    stamp = os.path.join(OBJ_DIR, "digest.txt")
    dig = _digest()
    if not force and os.path.exists(OUT) and os.path.exists(stamp) and open(stamp).read() == dig:
        return OUT
    os.makedirs(OBJ_DIR, exist_ok=True)
    nvcc = nvcc_path()
    flags = ["-O3", "-std=c++17", "-lineinfo", "-Xcompiler", "-fPIC", "-I", CSRC] + ARCH
    if verbose:
        flags += ["-Xptxas", "-v"]

    headers = hashlib.sha256()
    for f in sorted(os.listdir(CSRC)):
        if not f.endswith(".cu"):
            with open(os.path.join(CSRC, f), "rb") as fh:
                headers.update(f.encode() + fh.read())

    def compile_one(src: str) -> str:
        obj = os.path.join(OBJ_DIR, os.path.basename(src)[:-3] + ".o")
        fast = [] if os.path.basename(src) in PRECISE else ["--use_fast_math"]
        with open(src, "rb") as fh:
            made_of = hashlib.sha256(headers.digest() + fh.read() + " ".join([nvcc] + flags + fast).encode()).hexdigest()
        if not force and os.path.exists(obj) and os.path.exists(obj + ".txt") and open(obj + ".txt").read() == made_of:
            return obj
        cmd = [nvcc] + flags + fast + ["-c", src, "-o", obj]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if verbose or r.returncode != 0:
            sys.stderr.write(f"$ {' '.join(cmd)}\n{r.stdout}{r.stderr}\n")
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src}")
        with open(obj + ".txt", "w") as f:
            f.write(made_of)
        return obj

    with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 4)) as ex:
        objs = list(ex.map(compile_one, sources()))
    cmd = [nvcc, "-shared", "-o", OUT] + objs + ARCH + ["-lcudart"]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        sys.stderr.write(r.stdout + r.stderr)
        raise RuntimeError("link failed")
    with open(stamp, "w") as f:
        f.write(dig)
    return OUT


if __name__ == "__main__":
    print(build(verbose="-v" in sys.argv, force="-f" in sys.argv or "-v" in sys.argv))
