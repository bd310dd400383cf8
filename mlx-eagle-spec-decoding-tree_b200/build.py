"""Build the CUDA libraries in-tree with nvcc for sm_100a: ``libb200eagle.so`` (``csrc/*.cu``: 4-bit Llama/Qwen2 models,
tree decoding) and ``libb200hybrid.so`` (``csrc/hybrid/*.cu``: layer-list decoders)."""
from __future__ import annotations

import fcntl
import glob
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libb200eagle.so")
HYBRID_LIB = os.path.join(HERE, "libb200hybrid.so")
LIBS = ("eagle", "hybrid")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-Wall", "--threads", "0", "-shared",
]


def _library(name: str):
    """(output path, sources, headers) of a library."""
    common = glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(ROOT, "include", "*.h"))
    if name == "eagle":
        return LIB, sorted(glob.glob(os.path.join(CSRC, "*.cu"))), common
    if name == "hybrid":
        d = os.path.join(CSRC, "hybrid")
        return HYBRID_LIB, sorted(glob.glob(os.path.join(d, "*.cu"))), common + glob.glob(os.path.join(d, "*.cuh"))
    raise KeyError(name)


def sources() -> list[str]:
    return _library("eagle")[1]


def needs_build(name: str = "eagle") -> bool:
    out, srcs, headers = _library(name)
    if not os.path.exists(out):
        return True
    return any(os.path.getmtime(d) > os.path.getmtime(out) for d in srcs + headers)


def build(force: bool = False, verbose: bool = False, libs=LIBS) -> str:
    """Compile the named libraries where their sources are newer (each from its own sources only); returns the path of
    the last one.  Safe to call from several processes: a lock file serialises them, the result is moved into place."""
    for name in libs:
        out, srcs, _ = _library(name)
        if not force and not needs_build(name):
            continue
        with open(out + ".lock", "w") as lock:
            fcntl.flock(lock, fcntl.LOCK_EX)
            if not force and not needs_build(name):
                continue
            part = f"{out}.{os.getpid()}.tmp.so"
            cmd = [os.environ.get("NVCC") or shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"] + NVCC_FLAGS + ["-I", os.path.join(ROOT, "include"), "-I", CSRC]
            if verbose:
                cmd += ["-Xptxas", "-v"]
            res = subprocess.run(cmd + ["-o", part] + srcs, capture_output=True, text=True)
            if res.returncode != 0:
                sys.stderr.write(res.stdout + res.stderr)
                raise RuntimeError(f"nvcc failed building {os.path.basename(out)}")
            if verbose:
                sys.stderr.write(res.stderr)
            os.replace(part, out)
    return out


if __name__ == "__main__":
    print(build(force=True, verbose="-v" in sys.argv))
