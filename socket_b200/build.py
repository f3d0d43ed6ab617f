"""In-tree build of the CUDA libraries (sm_100a only).

    python -m socket_b200.build [--force] [--verbose] [library ...]

Two C-ABI shared libraries, compiled from `csrc/*.cu` with nvcc for `arch=compute_100a,code=sm_100a`:

* `step`   `socket_b200/libsocket_b200.so`         the sparse-attention step (`include/socket_b200.h`)
* `blocks` `socket_b200/libsocket_b200_blocks.so`  decoder building blocks (`include/socket_b200_blocks.h`)

A model compiles the libraries it uses and no more.  nvcc cross-compiles, so this runs on machines
without a GPU.
"""
from __future__ import annotations

import fcntl
import glob
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

PKG = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG, "csrc")
OBJ = os.path.join(CSRC, "obj")
LIB = os.path.join(PKG, "libsocket_b200.so")
BLOCKS_LIB = os.path.join(PKG, "libsocket_b200_blocks.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-lineinfo", "-std=c++17",
         "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
         "--expt-relaxed-constexpr"]
LIBRARIES = {"step": LIB, "blocks": BLOCKS_LIB}
BLOCK_SOURCES = ("abi_blocks", "attn_decode", "attn_prefill", "attn_rows", "latent", "mlstm", "mlstm_tc",
                 "recurrence_chunks", "residual", "rotary_rows", "ssm")
SHARED_SOURCES = ("host",)


def _sources(library: str):
    def member(name):
        return name in SHARED_SOURCES or (name in BLOCK_SOURCES) == (library == "blocks")
    return [s for s in sorted(glob.glob(os.path.join(CSRC, "*.cu"))) if member(os.path.basename(s)[:-3])]


def _deps():
    return glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(PKG, "..", "include", "*.h"))


def _stale(target, sources):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(s) > t for s in sources)


def build(force: bool = False, verbose: bool = False, libraries=("step", "blocks")) -> str:
    """Brings the named libraries up to date; returns the path of the first."""
    os.makedirs(OBJ, exist_ok=True)
    with open(os.path.join(OBJ, ".lock"), "w") as lock:      # one builder at a time
        fcntl.flock(lock, fcntl.LOCK_EX)
        _build_locked(force, verbose, libraries)
    return LIBRARIES[libraries[0]]


def _build_locked(force: bool, verbose: bool, libraries) -> None:
    deps = _deps()
    jobs, objs = {}, {}
    for library in libraries:
        objs[library] = []
        for src in _sources(library):
            obj = os.path.join(OBJ, os.path.basename(src)[:-3] + ".o")
            objs[library].append(obj)
            if force or _stale(obj, [src] + deps):
                cmd = [NVCC, *FLAGS, "-c", src, "-o", obj]
                if verbose:
                    cmd.insert(1, "-Xptxas")
                    cmd.insert(2, "-v")
                jobs[obj] = cmd

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        return cmd, r

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        for cmd, r in ex.map(run, jobs.values()):
            if verbose or r.returncode != 0:
                sys.stderr.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
            if r.returncode != 0:
                raise RuntimeError(f"nvcc failed on {cmd[-3]}")
    for library in libraries:
        target = LIBRARIES[library]
        if force or _stale(target, objs[library]):
            cmd = [NVCC, "-shared", "-o", target, *objs[library], "-gencode", "arch=compute_100a,code=sm_100a",
                   "-Xcompiler", "-fPIC"]
            r = subprocess.run(cmd, capture_output=True, text=True)
            if r.returncode != 0:
                sys.stderr.write(r.stdout + r.stderr)
                raise RuntimeError("link failed")


if __name__ == "__main__":
    named = [a for a in sys.argv[1:] if not a.startswith("-")]
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, libraries=named or ("step", "blocks")))
