"""Build ``libb2kv.so`` (the C-ABI CUDA library) in-tree with nvcc for sm_100a.

``python llm-experiments_b200/build.py [--force] [--verbose] [--serve]``.  The library has no
dependency on torch or Python: it is loaded with ctypes.  Sources are compiled to
objects in parallel and linked with the static CUDA runtime.

``--serve`` builds ``libb2kv_serve.so`` instead: only what models with a 32-bit residual stream are served with, a
fraction of the compile time (the decode-attention and prefill variants of the reference path take most of it).  It is
loaded where the whole library has not been built.
"""
from __future__ import annotations

import concurrent.futures
import os
import pathlib
import subprocess
import sys

PKG = pathlib.Path(__file__).resolve().parent
CSRC = PKG / "csrc"
INCLUDE = PKG.parent / "include"
OUT = PKG / "libb2kv.so"
SERVE_OUT = PKG / "libb2kv_serve.so"
OBJ_DIR = PKG / "build"
SERVE_SOURCES = ("api", "append", "gemm", "gla", "gla_chunked", "gqa", "gqa_decode_tc", "latent", "latent_decode_tc", "latent_prefill", "linear", "linear_rows", "moe", "rows",
                 "step_tail")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]


def _nvcc() -> str:
    cand = os.environ.get("NVCC") or "/usr/local/cuda/bin/nvcc"
    return cand if os.path.exists(cand) else "nvcc"


def sources(serve: bool = False):
    return [f for f in sorted(CSRC.glob("*.cu")) if not serve or f.stem in SERVE_SOURCES]


def _newest_input() -> float:
    files = list(CSRC.glob("*.cu")) + list(CSRC.glob("*.cuh")) + list(INCLUDE.glob("*.h"))
    return max(f.stat().st_mtime for f in files)


def up_to_date(out: pathlib.Path = OUT) -> bool:
    return out.exists() and out.stat().st_mtime >= _newest_input()


def build(force: bool = False, verbose: bool = False, serve: bool = False) -> pathlib.Path:
    out = SERVE_OUT if serve else OUT
    if not force and up_to_date(out):
        return out
    OBJ_DIR.mkdir(exist_ok=True)
    extra = ["-Xptxas", "-v"] if verbose else []

    def compile_one(src: pathlib.Path) -> pathlib.Path:
        obj = OBJ_DIR / (src.stem + ".o")
        cmd = [_nvcc(), *NVCC_FLAGS, *extra, "-I", str(INCLUDE), "-c", str(src), "-o", str(obj)]
        res = subprocess.run(cmd, capture_output=True, text=True)
        if verbose or res.returncode != 0:
            sys.stderr.write(res.stdout + res.stderr)
        if res.returncode != 0:
            raise RuntimeError(f"nvcc failed on {src.name}")
        return obj

    with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 1)) as pool:
        objs = list(pool.map(compile_one, sources(serve)))
    link = [_nvcc(), "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", str(out), *map(str, objs)]
    subprocess.run(link, check=True)
    return out


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, serve="--serve" in sys.argv))
