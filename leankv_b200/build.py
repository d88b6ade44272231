"""Builds the C-ABI libraries in-tree with nvcc for sm_100a.

Usage: ``python -m leankv_b200.build [--force] [--verbose]``. ``libleankv_b200.so`` holds the TEAL and
TurboQuant kernels, ``libleankv_mixers.so`` the token mixers and dense layers; a model loads (and on
first use builds) the one it needs. The libraries are placed next to this file so that they travel
with a snapshot of the source tree. nvcc cross-compiles without a GPU present.
"""

from __future__ import annotations

import fcntl
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

PKG_DIR = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(PKG_DIR)
CSRC = os.path.join(PKG_DIR, "csrc")
BUILD_DIR = os.path.join(PKG_DIR, "build")

# library -> sources; capi.cu (status codes, device queries) is linked into each
LIBRARIES = {
    "libleankv_b200.so": ["capi.cu", "teal_gemv.cu", "tq_quantize.cu", "tq_attn.cu", "decoder_ops.cu",
                          "decode_fused.cu"],
    "libleankv_mixers.so": ["capi.cu", "dense_gemv.cu", "stream_ops.cu", "window_pool.cu",
                            "window_pool_tile.cu", "time_mix.cu", "mixer_step.cu", "causal_rows.cu", "causal_tile.cu",
                            "causal_step.cu"],
}
LIB_PATH = os.path.join(PKG_DIR, "libleankv_b200.so")
MIXERS_PATH = os.path.join(PKG_DIR, "libleankv_mixers.so")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "-I", os.path.join(ROOT, "include"),
    "-I", CSRC,
]


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found: the sm_100a kernels cannot be built")
    return exe


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def build_library(name: str, force: bool = False, verbose: bool = False) -> str:
    """Compile the sources of one library and link it. Returns its path. Safe to call from several
    processes at once (one builds, the others wait)."""
    os.makedirs(BUILD_DIR, exist_ok=True)
    nvcc = _nvcc()
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    headers += [os.path.join(ROOT, "include", f) for f in os.listdir(os.path.join(ROOT, "include"))]
    sources = LIBRARIES[name]
    target = os.path.join(PKG_DIR, name)

    def compile_one(src: str) -> str:
        path = os.path.join(CSRC, src)
        obj = os.path.join(BUILD_DIR, src.replace(".cu", ".o"))
        if force or _stale(obj, [path] + headers):
            cmd = [nvcc, *NVCC_FLAGS, "-c", path, "-o", obj]
            if verbose:
                cmd.insert(1, "-Xptxas")
                cmd.insert(2, "-v")
            res = subprocess.run(cmd, capture_output=True, text=True)
            if verbose or res.returncode != 0:
                sys.stderr.write(f"--- {src}\n{res.stdout}{res.stderr}")
            if res.returncode != 0:
                raise RuntimeError(f"nvcc failed on {src}")
        return obj

    with open(os.path.join(BUILD_DIR, "lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        with ThreadPoolExecutor(max_workers=min(8, len(sources))) as pool:
            objs = list(pool.map(compile_one, sources))
        if force or _stale(target, objs):
            cmd = [nvcc, "-shared", "-o", target, *objs, "-gencode", "arch=compute_100a,code=sm_100a"]
            res = subprocess.run(cmd, capture_output=True, text=True)
            if res.returncode != 0:
                sys.stderr.write(res.stdout + res.stderr)
                raise RuntimeError(f"link of {name} failed")
    return target


def build(force: bool = False, verbose: bool = False) -> str:
    """Build every library. Returns the path of ``libleankv_b200.so``."""
    for name in LIBRARIES:
        build_library(name, force, verbose)
    return LIB_PATH


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
