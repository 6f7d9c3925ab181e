"""Build the native libraries in-tree.

``lib/liblmoe.so``       CUDA kernels for sm_100a (every ``csrc/*.cu``), plain C ABI, loaded with ctypes
``lib/liblmoe_host.so``  host-side C++ helpers (``csrc/host/*.cpp``)

``nvcc`` cross-compiles without a GPU.  Objects are rebuilt only when a source or header is newer.
Run ``python -m linear_moe_b200.build`` or call :func:`build_all`.
"""
from __future__ import annotations

import glob
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

ROOT = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(ROOT, "csrc")
LIB = os.path.join(ROOT, "lib")
OBJ = os.path.join(ROOT, "build")

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "--use_fast_math",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden"]
# sources whose fp32 instantiations serve models in true 32-bit: IEEE division and the accurate exp / tanh
PRECISE = {"chunk_attn.cu", "parallel_block.cu", "packed_attn.cu", "sandwich_block.cu", "moe_rows.cu", "post_norm.cu", "retention.cu", "ssd.cu",
           "delta_rule.cu"}
# what serving a model of the listed kind needs (``build_serving``); everything else is training, communication and fp8
SERVING = {"parallel_block": ("chunk_attn.cu", "chunk_attn_step.cu", "chunk_attn_tc.cu", "parallel_block.cu", "gemm_dense.cu", "gemm_skinny.cu"),
           "sandwich_block": ("packed_attn.cu", "packed_attn_step.cu", "packed_attn_tc.cu", "latent_step.cu", "moe_rows.cu", "sandwich_block.cu",
                              "parallel_block.cu", "gemm_dense.cu", "gemm_grouped.cu", "gemm_skinny.cu"),
           "post_norm_block": ("packed_attn.cu", "packed_attn_tc.cu", "talk_step.cu", "retention.cu", "retention_tc.cu", "post_norm.cu", "sandwich_block.cu",
                               "parallel_block.cu", "gemm_dense.cu", "gemm_skinny.cu"),
           "zelinex": ("packed_attn.cu", "packed_attn_step.cu", "packed_attn_tc.cu", "ssd.cu", "ssd_tc.cu", "delta_rule.cu", "delta_rule_tc.cu", "moe_rows.cu",
                       "sandwich_block.cu", "parallel_block.cu", "gemm_dense.cu", "gemm_grouped.cu", "gemm_skinny.cu")}


def _nvcc() -> str:
    cand = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(cand):
        raise RuntimeError("nvcc not found")
    return cand


def _newer(target: str, deps) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _run(cmd):
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("command failed: " + " ".join(cmd) + "\n" + r.stdout + r.stderr)
    return r.stdout + r.stderr


def _flags(src: str):
    return [f for f in NVCC_FLAGS if not (f == "--use_fast_math" and os.path.basename(src) in PRECISE)]


def build_cuda(verbose: bool = False, extra_flags=(), sources=None, name: str = "liblmoe.so") -> str:
    """``lib/<name>`` from ``sources`` (file names in ``csrc``; default: all of them)."""
    os.makedirs(LIB, exist_ok=True)
    os.makedirs(OBJ, exist_ok=True)
    srcs = sorted(glob.glob(os.path.join(CSRC, "*.cu"))) if sources is None else [os.path.join(CSRC, s) for s in sources]
    hdrs = glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h"))
    nvcc = _nvcc()
    objs, jobs = [], []
    for s in srcs:
        o = os.path.join(OBJ, os.path.basename(s)[:-3] + ".o")
        objs.append(o)
        if _newer(o, [s] + hdrs):
            jobs.append([nvcc, *_flags(s), *extra_flags, "-I", CSRC, "-c", s, "-o", o])
    with ThreadPoolExecutor(max_workers=min(8, max(len(jobs), 1))) as ex:
        for out in ex.map(_run, jobs):
            if verbose and out.strip():
                print(out)
    so = os.path.join(LIB, name)
    if jobs or _newer(so, objs):
        _run([nvcc, "-shared", "-o", so, *objs, "-lcudart"])
    return so


def build_serving(kind: str) -> str:
    """The kernel library for serving one kind of model (a key of ``SERVING``): the full ``liblmoe.so`` when it is there and
    newer than its sources, else a library of the sources that kind needs, compiled on the first call.  Processes that start
    together build once (a lock file), and a finished library replaces the old one in one step."""
    import fcntl
    full = os.path.join(LIB, "liblmoe.so")
    srcs = glob.glob(os.path.join(CSRC, "*.cu")) + glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h"))
    if not _newer(full, srcs):
        return full
    os.makedirs(LIB, exist_ok=True)
    with open(os.path.join(LIB, ".build.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return build_cuda(sources=SERVING[kind], name=f"liblmoe_{kind}.so")


def build_host(verbose: bool = False, sanitize: bool = False, out_dir: str = None) -> str:
    """``sanitize``: an AddressSanitizer + UndefinedBehaviorSanitizer build (``liblmoe_host_asan.so``) for the tests that
    run the host helpers under the sanitizers; it is loaded into a process that preloads the ASan runtime."""
    out_dir = out_dir or LIB
    os.makedirs(out_dir, exist_ok=True)
    srcs = sorted(glob.glob(os.path.join(CSRC, "host", "*.cpp")))
    so = os.path.join(out_dir, "liblmoe_host_asan.so" if sanitize else "liblmoe_host.so")
    if srcs and _newer(so, srcs):
        flags = ["-O1", "-g", "-fsanitize=address,undefined", "-fno-sanitize-recover=all", "-fno-omit-frame-pointer"] \
            if sanitize else ["-O3"]
        _run(["g++", *flags, "-std=c++17", "-fPIC", "-shared", "-pthread", "-o", so, *srcs])
    return so


def build_all(verbose: bool = False):
    return build_cuda(verbose), build_host(verbose)


if __name__ == "__main__":
    print(build_all(verbose="-v" in sys.argv))
