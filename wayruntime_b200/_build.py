"""Build libwr_cuda.so in-tree with nvcc for sm_100a (cross-compiles without a GPU)."""
from __future__ import annotations

import fcntl
import hashlib
import os
import shutil
import subprocess
import tempfile
from concurrent.futures import ThreadPoolExecutor

PKG = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG, "csrc")
LIB_DIR = os.path.join(PKG, "lib")
LIB_PATH = os.path.join(LIB_DIR, "libwr_cuda.so")
STAMP_PATH = LIB_PATH + ".sources"          # digest of what the library was built from
INCLUDE = os.path.join(os.path.dirname(PKG), "include")

SOURCES = ["kv_cache.cu", "attn_decode.cu", "attn_decode_static.cu", "attn_prefill.cu", "attn_exchange.cu",
           "model_glue.cu", "attn_step_small.cu", "gemv.cu", "gemm_bf16.cu", "gemm_skinny.cu", "mixers.cu", "latent.cu", "attn_latent.cu",
           "moe.cu", "model_mixed.cu"]
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
]


def _digest() -> str:
    h = hashlib.sha256(" ".join(NVCC_FLAGS).encode())
    for path in sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC)) + [os.path.join(INCLUDE, "wr_cuda.h")]:
        with open(path, "rb") as f:
            h.update(os.path.basename(path).encode() + b"\0" + f.read())
    return h.hexdigest()


def _stale() -> bool:
    if not os.path.exists(LIB_PATH):
        return True
    try:
        with open(STAMP_PATH) as f:
            return f.read().strip() != _digest()
    except OSError:
        return True


def build(force: bool = False, verbose: bool = False) -> str:
    """Compile the CUDA sources into wayruntime_b200/lib/libwr_cuda.so (one nvcc per source, in parallel).
    Safe to call from several processes at once: one builds, the others wait and find it done."""
    if not force and not _stale():
        return LIB_PATH
    os.makedirs(LIB_DIR, exist_ok=True)
    with open(os.path.join(LIB_DIR, ".build.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and not _stale():
            return LIB_PATH
        nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
        digest = _digest()
        tmp = tempfile.mkdtemp(dir=LIB_DIR)
        try:
            def run(cmd):
                res = subprocess.run(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
                if res.returncode != 0:
                    raise RuntimeError(f"nvcc failed:\n{res.stdout}")
                if verbose:
                    print(res.stdout)

            def compile_one(src):
                obj = os.path.join(tmp, src[:-3] + ".o")
                run([nvcc, *NVCC_FLAGS, "-I", INCLUDE, "-I", CSRC, *(["-Xptxas", "-v"] if verbose else []),
                     "-c", os.path.join(CSRC, src), "-o", obj])
                return obj

            with ThreadPoolExecutor(max(1, min(len(SOURCES), os.cpu_count() or 1))) as pool:
                objs = list(pool.map(compile_one, SOURCES))
            so = os.path.join(tmp, "libwr_cuda.so")
            run([nvcc, *NVCC_FLAGS, "-shared", *objs, "-o", so])
            os.replace(so, LIB_PATH)
            with open(os.path.join(tmp, "stamp"), "w") as f:
                f.write(digest)
            os.replace(os.path.join(tmp, "stamp"), STAMP_PATH)
        finally:
            shutil.rmtree(tmp, ignore_errors=True)
    return LIB_PATH


DROPIN_PATH = os.path.join(LIB_DIR, "libwayruntime_b200.so")


def build_dropin(ref_root: str) -> str | None:
    """Link lib/libwayruntime_b200.so: the reference library (compiled from the
    checkout at `ref_root`, unmodified) with this package's session objects and
    engine gate in place of its session.c / batch.c / engine entry points.
    Returns None when there is no checkout (the GPU box uses the prebuilt file)."""
    if not os.path.exists(os.path.join(ref_root, "src", "core", "kernels.c")):
        return None
    build()
    res = subprocess.run(["make", "-C", os.path.join(PKG, "host"), f"REF={ref_root}"],
                         stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"drop-in link failed:\n{res.stdout}")
    return DROPIN_PATH
