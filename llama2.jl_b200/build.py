"""In-tree build of the CUDA library for sm_100a (cross-compiles without a GPU)."""
import fcntl
import hashlib
import os
import shutil
import subprocess
from concurrent.futures import ThreadPoolExecutor

_HERE = os.path.dirname(os.path.abspath(__file__))
SOURCES = ["csrc/api.cu", "csrc/stack.cu", "csrc/stack_config.cpp", "csrc/safetensors.cpp", "csrc/gguf_reader.cpp", "csrc/tokenizer.cpp"]
HEADERS = ["csrc/common.cuh", "csrc/kquants.cuh", "csrc/fused_matvec.cuh", "csrc/attention.cuh", "csrc/sampling.cuh",
           "csrc/small_ops.cuh", "csrc/token_kernel.cuh", "csrc/kq_gemm.cuh", "csrc/prefill_ops.cuh", "csrc/gguf_reader.h", "csrc/host_common.h",
           "csrc/tcgen05.cuh", "csrc/json.h", "csrc/safetensors.h", "csrc/stack_config.h", "csrc/stack.h", "csrc/dense_ops.cuh",
           "csrc/dense_matvec.cuh", "csrc/dense_gemm.cuh", "csrc/stack_rows.cuh", "csrc/cache_scan.cuh", "csrc/latent_attention.cuh",
           "csrc/head_attention.cuh", "csrc/head_prefill.cuh", "csrc/mlstm.cuh", "csrc/mlstm_prefill.cuh", "csrc/latent_prefill.cuh",
           "../include/llama2_b200.h"]
OUTPUT = os.path.join(_HERE, "libllama2_b200.so")
SYNTH_OUTPUT = os.path.join(_HERE, "libl2b_synth.so")  # test support: seeded synthetic data, plain C++
BUILD_DIR = os.path.join(_HERE, "build")
STAMP = os.path.join(BUILD_DIR, "library.sha256")
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC"]


def _nvcc():
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", shutil.which("nvcc")):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc was not found (set NVCC)")


def _digest():
    """What the library is built from: contents of the sources and the flags (file times do not survive a copy)."""
    h = hashlib.sha256(" ".join(NVCC_FLAGS).encode())
    for f in SOURCES + HEADERS:
        with open(os.path.join(_HERE, f), "rb") as fp:
            h.update(f.encode() + b"\0" + fp.read())
    return h.hexdigest()


def needs_build():
    try:
        with open(STAMP) as f:
            return not os.path.exists(OUTPUT) or f.read().strip() != _digest()
    except OSError:
        return True


def build_synth(force=False):
    src = os.path.join(_HERE, "csrc/synth.cpp")
    if force or not os.path.exists(SYNTH_OUTPUT) or os.path.getmtime(src) > os.path.getmtime(SYNTH_OUTPUT):
        subprocess.run([os.environ.get("CXX", "g++"), "-O2", "-std=c++17", "-fPIC", "-shared", "-pthread", "-o", SYNTH_OUTPUT, src], check=True)
    return SYNTH_OUTPUT


def build_measure():
    """A second library with the measurement aids compiled in (-DL2B_MEASURE): time stamps inside the kernels, switches that
    skip parts of them.  Not the product: load it with L2B_LIBRARY=<path> for your own measurements."""
    out = os.path.join(_HERE, "libllama2_b200_measure.so")
    subprocess.run([_nvcc()] + NVCC_FLAGS + ["-shared", "-DL2B_MEASURE", "-o", out] + [os.path.join(_HERE, s) for s in SOURCES], check=True)
    return out


def build_library(force=False, verbose=False):
    """The product library alone: every source to an object of its own, side by side, then one link.  Compiler output goes to
    standard error.  Safe against a second process building the same tree."""
    os.makedirs(BUILD_DIR, exist_ok=True)
    with open(os.path.join(BUILD_DIR, "lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and not needs_build():
            return OUTPUT
        digest = _digest()

        def compile_one(src):
            obj = os.path.join(BUILD_DIR, os.path.basename(src) + ".o")
            extra = ["-Xptxas", "-v"] if verbose and src.endswith(".cu") else []
            subprocess.run([_nvcc()] + NVCC_FLAGS + extra + ["-c", "-o", obj, os.path.join(_HERE, src)], check=True, stdout=2)
            return obj
        with ThreadPoolExecutor(len(SOURCES)) as pool:
            objs = list(pool.map(compile_one, SOURCES))
        tmp = OUTPUT + ".tmp"
        subprocess.run([_nvcc()] + NVCC_FLAGS + ["-shared", "-o", tmp] + objs, check=True, stdout=2)
        os.replace(tmp, OUTPUT)
        with open(STAMP, "w") as f:
            f.write(digest)
    return OUTPUT


def build(force=False, verbose=False):
    build_synth(force)
    return build_library(force, verbose)


if __name__ == "__main__":
    print(build(force=True, verbose=True))
