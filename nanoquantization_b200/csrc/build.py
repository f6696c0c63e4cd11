"""Build the libraries (sm_100a) in-tree with nvcc.  Cross-compiles without a GPU.

Three shared objects: ``libnqb200.so`` (the W4A16 linears, their elementwise neighbours and the peer all-reduce),
``libnqb200_mixers.so`` (the sequence-mixing kernels) and ``libnqb200_moe.so`` (mixtures of experts).  They are built separately so that a model compiles only what
it uses; the sources of a library are compiled side by side."""
from __future__ import annotations

import os
import subprocess
import sys
import tempfile
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(os.path.dirname(HERE))
LIB_DIR = os.path.join(os.path.dirname(HERE), "lib")
LIB_PATH = os.path.join(LIB_DIR, "libnqb200.so")
MIXERS_PATH = os.path.join(LIB_DIR, "libnqb200_mixers.so")
MOE_PATH = os.path.join(LIB_DIR, "libnqb200_moe.so")
SOURCES = ["api.cu", "unpack_dequant.cu", "gemm_decode.cu", "gemm_stream.cu", "gemm_umma_prefill.cu", "gemm_umma_pair.cu", "quantize_pack.cu", "fused_elementwise.cu", "peer_allreduce.cu"]
HEADERS = ["common.cuh", "tma_utils.cuh", "umma_utils.cuh", os.path.join(ROOT, "include", "nqb200.h")]
MIXER_SOURCES = ["mixer_norm.cu", "mixer_attention.cu", "mixer_recurrent.cu", "mixer_dense.cu", "mixer_decode.cu", "mixer_prefill.cu", "mixer_attention_umma.cu", "mixer_gla.cu"]
MIXER_HEADERS = ["common.cuh", "mixers.cuh", "mma_utils.cuh", "tma_utils.cuh", "umma_utils.cuh", os.path.join(ROOT, "include", "nqb200.h"), os.path.join(ROOT, "include", "nqb200_mixers.h")]
MOE_SOURCES = ["moe_route.cu", "moe_experts.cu", "moe_umma.cu"]
MOE_HEADERS = MIXER_HEADERS + ["moe.cuh", os.path.join(ROOT, "include", "nqb200_moe.h")]
LIBRARIES = {LIB_PATH: (SOURCES, HEADERS), MIXERS_PATH: (MIXER_SOURCES, MIXER_HEADERS), MOE_PATH: (MOE_SOURCES, MOE_HEADERS)}


def _stale(path: str = LIB_PATH) -> bool:
    if not os.path.exists(path):
        return True
    t = os.path.getmtime(path)
    sources, headers = LIBRARIES[path]
    return any(os.path.getmtime(os.path.join(HERE, d)) > t for d in sources + headers)


def build_library(path: str, force: bool = False, verbose: bool = False) -> str:
    """One of the libraries; returns its path.  The finished file is moved into place, so that a process that loads
    it while another builds sees a whole library."""
    if not force and not _stale(path):
        return path
    os.makedirs(LIB_DIR, exist_ok=True)
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    sources, _ = LIBRARIES[path]
    flags = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC",
             "-I", os.path.join(ROOT, "include"), "-I", HERE] + (["-Xptxas", "-v"] if verbose else [])
    with tempfile.TemporaryDirectory() as tmp:
        objects = [os.path.join(tmp, s.replace(".cu", ".o")) for s in sources]

        def compile_one(job):
            src, obj = job
            subprocess.check_call([nvcc, *flags, "-c", os.path.join(HERE, src), "-o", obj])
        with ThreadPoolExecutor(max_workers=min(len(sources), os.cpu_count() or 1)) as pool:
            list(pool.map(compile_one, zip(sources, objects)))
        part = f"{path}.{os.getpid()}.part"
        subprocess.check_call([nvcc, *flags, "-shared", *objects, "-o", part])
        os.replace(part, path)
    return path


def build(force: bool = False, verbose: bool = False) -> str:
    for path in LIBRARIES:
        build_library(path, force, verbose)
    return LIB_PATH


if __name__ == "__main__":
    build(force=True, verbose="-v" in sys.argv)
    print("\n".join(LIBRARIES))
