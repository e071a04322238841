"""Build the sm_100a kernel library in-tree.

``python -m slime_b200.ops.build`` compiles every ``csrc/*.cu`` with
``nvcc -gencode arch=compute_100a,code=sm_100a -lineinfo`` (objects in parallel)
and links ``slime_b200/ops/_kernels.so``. The library exposes a plain C ABI that
``slime_b200.ops._lib`` binds with ctypes, so no PyTorch headers are compiled.
nvcc cross-compiles without a GPU.
"""

from __future__ import annotations

import concurrent.futures
import hashlib
import os
import shutil
import subprocess
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
CSRC = os.path.join(ROOT, "csrc")
OUT = os.path.join(ROOT, "slime_b200", "ops", "_kernels.so")
OBJ_DIR = os.path.join(ROOT, "build", "obj")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xptxas", "-v",
]  # fmt: skip
# extra compiler flags, e.g. SLIME_B200_NVCC_EXTRA="-DSB_WS_CHAIN_TIMING" for a measurement build
NVCC_FLAGS += os.environ.get("SLIME_B200_NVCC_EXTRA", "").split()


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found; the sm_100a kernels cannot be built")
    return exe


def _digest(paths) -> str:
    h = hashlib.sha256()
    for p in sorted(paths):
        with open(p, "rb") as f:
            h.update(os.path.basename(p).encode())  # not the absolute path: the tree may be copied elsewhere
            h.update(f.read())
    h.update(" ".join(NVCC_FLAGS).encode())
    return h.hexdigest()


def sources() -> list[str]:
    return sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cu"))


# Parts of the library that can be built on their own (``ensure``): a process that only serves layered models has no use for
# the training, fp8 and multi-GPU kernels, and a fresh checkout should not wait for them.
GROUPS = {"serve": ("gemm_sm100", "gemm_simt", "stream", "delta_rule", "linear_scan", "window_attn", "flash_window_sm100", "latent_sm100", "decode_attn_sm100", "paged_attn", "moe",
                    "quant", "elementwise", "sampling")}  # fmt: skip


def _headers() -> list[str]:
    return [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]


def _current(out: str, stamp: str, digest: str) -> bool:
    if not os.path.exists(out) or not os.path.exists(stamp):
        return False
    with open(stamp) as f:
        return f.read() == digest


def ensure(group: str) -> str:
    """Make sure the kernels of ``group`` are built and are what ``_lib`` loads: the whole library when it is there and
    current, otherwise a library of the group's sources alone (compiled now if needed)."""
    if _current(OUT, os.path.join(OBJ_DIR, "stamp.txt"), _digest(sources() + _headers())):
        return OUT
    from slime_b200.ops import _lib

    part = OUT.replace("_kernels.so", f"_kernels_{group}.so")
    path = build(srcs=[os.path.join(CSRC, f + ".cu") for f in GROUPS[group]], out=part)
    _lib.use_library(path)
    return path


def build(force: bool = False, verbose: bool = False, srcs: list[str] | None = None, out: str = OUT) -> str:
    """Compile ``srcs`` (default: every source) and link them into ``out``. Processes that build at the same time take turns."""
    import fcntl

    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(OBJ_DIR, "lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build(force, verbose, srcs or sources(), out)


def _build(force: bool, verbose: bool, srcs: list[str], out: str) -> str:
    stamp = os.path.join(OBJ_DIR, "stamp.txt" if out == OUT else os.path.basename(out) + ".stamp")
    digest = _digest(srcs + _headers())
    if not force and _current(out, stamp, digest):
        return out
    nvcc = _nvcc()

    def compile_one(src):
        obj = os.path.join(OBJ_DIR, os.path.basename(src) + ".o")
        cmd = [nvcc, *NVCC_FLAGS, "-I", CSRC, "-c", src, "-o", obj]
        res = subprocess.run(cmd, capture_output=True, text=True)
        log = res.stdout + res.stderr
        with open(obj + ".log", "w") as f:
            f.write(" ".join(cmd) + "\n" + log)
        if res.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src}:\n{log}")
        if verbose:
            print(log)
        return obj

    with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, len(srcs))) as pool:
        objs = list(pool.map(compile_one, srcs))
    tmp = f"{out}.{os.getpid()}.tmp"  # renamed when complete: a process that has the old file loaded keeps it
    link = [nvcc, "-shared", "-o", tmp, *objs, "-gencode", "arch=compute_100a,code=sm_100a"]
    res = subprocess.run(link, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError("link failed:\n" + res.stdout + res.stderr)
    os.replace(tmp, out)
    with open(stamp, "w") as f:
        f.write(digest)
    return out


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
