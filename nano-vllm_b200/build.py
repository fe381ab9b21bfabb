"""Build recipe of the CUDA library (libb200tp.so) for sm_100a.

nvcc cross-compiles without a GPU.  The library is built in-tree under
nano-vllm_b200/lib/ so that it travels with the source tree.
"""
from __future__ import annotations

import hashlib
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIBDIR = os.path.join(HERE, "lib")
LIB = os.path.join(LIBDIR, "libb200tp.so")
SOURCES = ["b2_ctx.cu", "b2_elementwise.cu", "b2_gemm.cu", "b2_gemm_f32.cu", "b2_streams.cu", "b2_attention.cu", "b2_linear_attn.cu",
           "b2_sandwich.cu", "b2_latent.cu", "b2_expanded.cu"]
HEADERS = ["b2_common.cuh", "b2_vec.cuh", "b2_mma.cuh", "b2_attn.cuh", os.path.join("..", "..", "include", "b200tp.h")]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17"]


def _stamp(sources: list[str]) -> str:
    h = hashlib.sha256()
    for name in sources + HEADERS:
        with open(os.path.join(CSRC, name), "rb") as f:
            h.update(f.read())
    h.update(" ".join(NVCC_FLAGS).encode())
    return h.hexdigest()


def build(force: bool = False, verbose: bool = False) -> str:
    """Compile every .cu into objects and link the shared library; returns its path."""
    os.makedirs(LIBDIR, exist_ok=True)
    stamp_file = os.path.join(LIBDIR, "build.stamp")
    stamp = _stamp(SOURCES)
    if not force and os.path.exists(LIB) and os.path.exists(stamp_file) and open(stamp_file).read() == stamp:
        return LIB
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    objs = []
    procs = []
    for src in SOURCES:
        obj = os.path.join(LIBDIR, src.replace(".cu", ".o"))
        objs.append(obj)
        mark = obj + ".stamp"
        if not force and not verbose and os.path.exists(obj) and os.path.exists(mark) and open(mark).read() == _stamp([src]):
            continue  # this source has not changed since its object was built
        cmd = [nvcc, *NVCC_FLAGS, "-Xcompiler", "-fPIC", "-c", os.path.join(CSRC, src), "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    for src, p in procs:
        out, _ = p.communicate()
        if verbose or p.returncode != 0:
            sys.stderr.write(out)
        if p.returncode != 0:
            raise RuntimeError(f"nvcc failed on {src}")
        with open(os.path.join(LIBDIR, src.replace(".cu", ".o.stamp")), "w") as f:
            f.write(_stamp([src]))
    cmd = [nvcc, "-shared", "-Wno-deprecated-gpu-targets", "-o", LIB, *objs, "-lcudart"]
    subprocess.check_call(cmd)
    with open(stamp_file, "w") as f:
        f.write(stamp)
    return LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
