"""Build the CUDA libraries in-tree with nvcc for sm_100a.

    python mirage_b200/build.py            # build what is older than its sources
    python mirage_b200/build.py --force
    python mirage_b200/build.py --only hybrid   # the C ABI library and one kernel family

libmpk_b200.so holds the C ABI, the task-graph compiler and the allocation-free attention entry point; the megakernel
instantiations are in one library per family beside it (decoder: transformer graphs; hybrid: graphs with recurrent or
extended-attention layers), loaded when a graph of the family is compiled.
"""
from __future__ import annotations

import fcntl
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB_DIR = os.path.join(HERE, "lib")
LIB_PATH = os.path.join(LIB_DIR, "libmpk_b200.so")
ABI_HEADER = os.path.join("..", "..", "include", "mpk_b200.h")
HOST_HEADERS = ["runtime_types.h", "task_graph.h", ABI_HEADER]
KERNEL_HEADERS = ["runtime_types.h", "device_utils.cuh", "megakernel.cuh", "hybrid_tasks.cuh"]
# library -> (sources, headers they depend on)
TARGETS = {
    "core": ("libmpk_b200.so", ["mpk_abi.cu", "task_graph.cpp", "shuffle_rows.cu", "noalloc_attention.cu"],
             HOST_HEADERS + ["device_utils.cuh"]),
    "decoder": ("libmpk_b200_decoder.so", ["decoder_kernels.cu"], KERNEL_HEADERS),
    "hybrid": ("libmpk_b200_hybrid.so", ["hybrid_kernels.cu", "hybrid_kernel_bf16.cu", "hybrid_kernel_bf16_wide.cu", "hybrid_kernel_f32.cu"],
               KERNEL_HEADERS + ["hybrid_kernels.h"]),
}
ARCH = ["-gencode", "arch=compute_100a,code=sm_100a"]
NVCC_FLAGS = [*ARCH, "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    return "nvcc"


def needs_build(target: str) -> bool:
    lib, sources, headers = TARGETS[target]
    path = os.path.join(LIB_DIR, lib)
    if not os.path.exists(path):
        return True
    t = os.path.getmtime(path)
    return any(os.path.getmtime(os.path.join(CSRC, f)) > t for f in sources + headers)


def _run(cmds):
    """All commands at once; the first failure is raised after every one has ended."""
    procs = [(c, subprocess.Popen(c)) for c in cmds]
    failed = [(c, p.returncode) for c, p in procs if p.wait() != 0]
    if failed:
        raise subprocess.CalledProcessError(failed[0][1], failed[0][0])


def build(force: bool = False, verbose: bool = False, only=None) -> str:
    """Build `only` these targets (default: all) where they are out of date; returns the C ABI library's path."""
    todo = [t for t in (only or TARGETS) if force or needs_build(t)]
    if not todo:
        return LIB_PATH
    os.makedirs(LIB_DIR, exist_ok=True)
    with open(os.path.join(LIB_DIR, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)              # two processes may start on a fresh checkout
        todo = [t for t in todo if force or needs_build(t)]
        compile_cmds, link_cmds = [], []
        for target in todo:
            lib, sources, _ = TARGETS[target]
            objs = []
            for src in sources:
                obj = os.path.join(LIB_DIR, src.rsplit(".", 1)[0] + ".o")
                cmd = [_nvcc(), *NVCC_FLAGS, "-x", "cu", "-c", os.path.join(CSRC, src), "-o", obj]
                if verbose:
                    cmd.insert(1, "-Xptxas=-v")
                compile_cmds.append(cmd)
                objs.append(obj)
            tmp = os.path.join(LIB_DIR, lib + ".tmp")
            link_cmds.append((tmp, os.path.join(LIB_DIR, lib),
                              [_nvcc(), *ARCH, "-shared", "-o", tmp, *objs, "-lcudart", "-ldl"]))
        _run(compile_cmds)
        _run([cmd for _, _, cmd in link_cmds])
        for tmp, path, _ in link_cmds:
            os.replace(tmp, path)
    return LIB_PATH


if __name__ == "__main__":
    names = [sys.argv[i + 1] for i, a in enumerate(sys.argv[:-1]) if a == "--only"]
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv, only=["core", *names] if names else None))
