"""Build libb200gpt.so (the sm_100a kernels + C ABI) in-tree with nvcc.

    python -m gpt_triton_b200.build [--force]

nvcc cross-compiles for sm_100a, so this works on a machine without a GPU.  Sources are compiled side by side, one
object file each; an object is rebuilt when its source or any header is newer.
"""

import os
import shutil
import subprocess
import sys
import tempfile
from concurrent.futures import ThreadPoolExecutor

PKG_DIR = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG_DIR, "csrc")
OBJ_DIR = os.path.join(PKG_DIR, "_obj")
LIB_PATH = os.path.join(PKG_DIR, "libb200gpt.so")
SOURCES = ["api.cu", "elementwise.cu", "gemm_sm100.cu", "linear_sm100.cu", "linear_f32.cu", "attention.cu", "attention_sm100.cu", "latent.cu",
           "latent_decode.cu", "lightning.cu", "stream.cu", "rotary.cu", "pair_attention.cu", "pair_attention_sm100.cu", "pair_decode.cu", "delta.cu", "delta_chunk.cu", "decode.cu", "ffn_static_scratch.cu", "selftest.cu"]
HEADERS = [os.path.join(CSRC, "common.cuh"), os.path.join(CSRC, "sm100_primitives.cuh"), os.path.join(CSRC, "gemm_sm100.cuh"),
           os.path.join(CSRC, "mma_sync.cuh"), os.path.join(CSRC, "attention_sm100.cuh"),
           os.path.join(os.path.dirname(PKG_DIR), "include", "b200_gpt.h")]
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC",
]


def _nvcc():
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found: libb200gpt.so cannot be built")
    return exe


def _newer(path, deps):
    """True if `path` exists and is not older than any of `deps`."""
    return os.path.exists(path) and all(os.path.getmtime(d) <= os.path.getmtime(path) for d in deps)


def is_stale():
    return not _newer(LIB_PATH, [os.path.join(CSRC, s) for s in SOURCES] + HEADERS)


def _run(cmd):
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError("nvcc failed:\n" + res.stdout + res.stderr)
    return res.stderr


def build(force=False, verbose=False):
    """Compile the library if it is missing or older than its sources; return its path."""
    if not force and not is_stale():
        return LIB_PATH
    nvcc = _nvcc()
    os.makedirs(OBJ_DIR, exist_ok=True)
    log = []

    def compile_one(name):
        src, obj = os.path.join(CSRC, name), os.path.join(OBJ_DIR, name[:-3] + ".o")
        if force or not _newer(obj, [src] + HEADERS):
            part = f"{obj}.{os.getpid()}.o"
            log.append(_run([nvcc, *NVCC_FLAGS, *(["-Xptxas", "-v"] if verbose else []), "-c", src, "-o", part]))
            os.replace(part, obj)
        return obj

    with ThreadPoolExecutor(max_workers=max(2, min(len(SOURCES), os.cpu_count() or 2))) as pool:
        objects = list(pool.map(compile_one, SOURCES))
    with tempfile.TemporaryDirectory(dir=OBJ_DIR) as tmp:  # linked aside and moved: a reader never sees half a library
        part = os.path.join(tmp, "lib.so")
        _run([nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", part, *objects])
        os.replace(part, LIB_PATH)
    if verbose:
        print("".join(log))
    return LIB_PATH


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
