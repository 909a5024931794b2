"""Build libnckv.so (all CUDA sources of this directory) for sm_100a with nvcc.

Usage:  python -m nanochat_b200.csrc.build [--verbose] [--force]
The shared library is written next to the package (nanochat_b200/libnckv.so); it is a build
artefact and is not tracked.
"""
import fcntl
import os
import subprocess
import sys
import tempfile
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
PKG = os.path.dirname(HERE)
OUT = os.path.join(PKG, "libnckv.so")
SOURCES = ["host.cu", "append.cu", "decode_attn.cu", "prefill_broadcast.cu", "lse_combine.cu",
           "prefill_attn.cu", "p2p_exchange.cu", "glue.cu", "flash_attn_bwd.cu", "host_step.cu",
           "recurrent.cu", "recurrent_f32.cu", "norm_mix.cu", "window_attn.cu", "hyper_norm.cu",
           "gated_linear.cu", "delta.cu", "delta_chunk.cu", "experts.cu", "experts_tc.cu"]
HEADERS = ["nckv_common.cuh", "vec_io.cuh", "tc05.cuh", "recurrent.cuh", "experts.cuh", os.path.join("..", "..", "include", "nckv.h")]


def _nvcc():
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    raise RuntimeError("nvcc not found")


def up_to_date():
    if not os.path.exists(OUT):
        return False
    t = os.path.getmtime(OUT)
    deps = [os.path.join(HERE, s) for s in SOURCES + HEADERS] + [os.path.abspath(__file__)]
    return all(os.path.getmtime(d) <= t for d in deps)


def _compile(cmd, verbose):
    res = subprocess.run(cmd, capture_output=True, text=True)
    if verbose or res.returncode != 0:
        sys.stderr.write(" ".join(cmd) + "\n" + res.stdout + res.stderr)
    return res.returncode


def build(verbose=False, force=False):
    """Compile the sources side by side, link them, and move the library into place in one step; several
    processes may call this at the same time."""
    if not force and up_to_date():
        return OUT
    with open(os.path.join(PKG, ".build.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and up_to_date():  # another process has built it meanwhile
            return OUT
        nvcc = _nvcc()
        flags = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC",
                 "-Xcompiler", "-fvisibility=hidden"] + (["-Xptxas", "-v"] if verbose else [])
        with tempfile.TemporaryDirectory(dir=PKG, prefix=".build-") as tmp:
            objs = [os.path.join(tmp, os.path.splitext(s)[0] + ".o") for s in SOURCES]
            jobs = [[nvcc] + flags + ["-c", "-o", o, os.path.join(HERE, s)] for s, o in zip(SOURCES, objs)]
            with ThreadPoolExecutor(max(1, min(len(jobs), os.cpu_count() or 1))) as pool:
                failed = any(list(pool.map(lambda cmd: _compile(cmd, verbose), jobs)))
            linked = os.path.join(tmp, os.path.basename(OUT))
            if failed or _compile([nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "--shared", "-o", linked] + objs, verbose):
                raise RuntimeError("nvcc failed building libnckv.so")
            os.replace(linked, OUT)
    return OUT


if __name__ == "__main__":
    build(verbose="--verbose" in sys.argv, force="--force" in sys.argv)
    print(OUT)
