"""Ahead-of-time build of the package's shared libraries for sm_100a with nvcc.

Two libraries with plain C ABIs and no torch dependency, built in-tree next to
the Python package: ``libmegaqwen_b200.so`` (the Qwen3-0.6B kernels,
include/megaqwen_b200.h) and ``libmegaqwen_hybrid.so`` (the layer-listed
decoder, include/megaqwen_hybrid.h).  Each is built alone when it is needed
alone; nvcc compiles the sources side by side and cross-compiles without a
GPU.  Run ``python -m megaqwen_b200.csrc.build``.
"""
from __future__ import annotations

import fcntl
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
PKG = os.path.dirname(HERE)
# library -> (sources, output)
LIBRARIES = {
    "qwen3": (["decode.cu", "decode_stream.cu", "prefill.cu", "ops.cu", "token_ops.cu"],
              os.environ.get("MQ_LIB_OUT") or os.path.join(PKG, "libmegaqwen_b200.so")),
    "hybrid": (["hy_linear.cu", "hy_gemv.cu", "hy_rows.cu", "hy_recurrence.cu", "hy_latent.cu", "hy_attention.cu", "hy_model.cu", "token_ops.cu"],
               os.path.join(PKG, "libmegaqwen_hybrid.so")),
}


def _stale(name: str) -> bool:
    sources, out = LIBRARIES[name]
    if not os.path.exists(out):
        return True
    t = os.path.getmtime(out)
    inc = os.path.join(os.path.dirname(PKG), "include")
    deps = [os.path.join(HERE, f) for f in os.listdir(HERE) if f in sources or f.endswith(".cuh")]
    deps += [os.path.join(inc, f) for f in os.listdir(inc)]
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False, name: str = "qwen3") -> str:
    """Build one library if it is missing or older than its sources; returns its path."""
    sources, out = LIBRARIES[name]
    if not force and not _stale(name):
        return out
    with open(out + ".lock", "w") as lock:        # two processes that both find it missing build it once
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and not _stale(name):
            return out
        nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
        cmd = [nvcc, "-std=c++17", "-O3", "-lineinfo", "-gencode", "arch=compute_100a,code=sm_100a", "--threads", "0",
               "-shared", "-Xcompiler", "-fPIC", "-o", out + ".new"]
        if verbose:
            cmd += ["-Xptxas", "-v"]
        cmd += os.environ.get("MQ_NVCC_FLAGS", "").split()
        cmd += [os.path.join(HERE, s) for s in sources]
        res = subprocess.run(cmd, capture_output=True, text=True)
        if res.returncode != 0:
            sys.stderr.write(res.stdout + res.stderr)
            raise RuntimeError(f"nvcc failed building {os.path.basename(out)}")
        os.replace(out + ".new", out)
        if verbose:
            sys.stderr.write(res.stderr)
    return out


def build_all(force: bool = False, verbose: bool = False) -> list:
    return [build(force, verbose, n) for n in LIBRARIES]


if __name__ == "__main__":
    names = [a for a in sys.argv[1:] if not a.startswith("-")] or list(LIBRARIES)
    for n in names:
        print(build(force=True, verbose="-v" in sys.argv, name=n))
