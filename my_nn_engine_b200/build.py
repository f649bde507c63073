"""Builds the sm_100a shared library ``libmynn_b200.so`` in-tree with nvcc.

    python -m my_nn_engine_b200.build [--force] [--verbose]

nvcc cross-compiles without a GPU.  The library links the static CUDA runtime only; NCCL is resolved with
dlopen at run time, so the file loads on a box without NCCL as long as tensor parallelism is not used.
"""
from __future__ import annotations

import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "libmynn_b200.so")
SOURCES = ["runtime.cu", "dequant_gemm.cu", "i8_gemm.cu", "gemv_lean.cu", "i8_gemm_prefill.cu", "w8a8.cu", "attention.cu", "attention_prefill.cu", "attention_prefill_tc.cu", "kv_int8.cu", "streaming_kv.cu", "glue.cu", "comm.cu", "tp_fused.cu", "model.cu",
           "layer_norm.cu", "short_conv.cu", "attention_window.cu", "rotary_append.cu", "latent_attention.cu", "mlstm.cu", "mlstm_tc.cu", "moe_route.cu", "dense_gemm.cu", "dense_gemm_tc.cu", "block_model.cu"]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC",
              "-DMYNN_COMPILED_ARCH=100"]


def _nvcc() -> str:
    cand = os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "bin", "nvcc")
    return cand if os.path.exists(cand) else "nvcc"


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False, defines: tuple = ()) -> str:
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    headers.append(os.path.join(HERE, "..", "include", "mynn_b200.h"))
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    objs, jobs = [], []
    for src in SOURCES:
        s = os.path.join(CSRC, src)
        o = os.path.join(objdir, src[:-3] + ".o")
        objs.append(o)
        if force or _stale(o, [s] + headers):
            cmd = [_nvcc()] + NVCC_FLAGS + ["-D" + d for d in defines] + (["-Xptxas", "-v"] if verbose else []) + ["-c", s, "-o", o]
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        if verbose or r.returncode:
            sys.stderr.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
        if r.returncode:
            raise RuntimeError(f"nvcc failed for {cmd[-3]}")

    with ThreadPoolExecutor(max_workers=6) as ex:
        list(ex.map(run, jobs))
    if force or jobs or _stale(OUT, objs):
        cmd = [_nvcc(), "-shared", "-o", OUT] + objs + ["-ldl"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
    return OUT


if __name__ == "__main__":
    # -DNAME[=value] arguments are passed to nvcc (e.g. -DMYNN_TUNING for the build with phase timestamps); use with --force
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, defines=tuple(a[2:] for a in sys.argv[1:] if a.startswith("-D"))))
