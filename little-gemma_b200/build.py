"""Build liblg_b200.so in-tree: host C (gcc) + sm_100a CUDA (nvcc), one shared library.

    python little-gemma_b200/build.py [--mtp-n 4] [--force] [--ptxas-v]

The library is compiled for sm_100a only; nvcc cross-compiles without a GPU.
"""
from __future__ import annotations

import argparse
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
INC = os.path.join(ROOT, "include")
HOST = os.path.join(HERE, "csrc", "host")
CUDA = os.path.join(HERE, "csrc", "cuda")
LIB = os.path.join(HERE, "liblg_b200.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")

HOST_SRC = ["lg_gguf.c", "lg_ckpt.c", "lg_quant.c", "lg_plan.c", "lg_setup.c", "lg_session.c"]
CUDA_SRC = {"lg_engine.cu": ["lg_engine.h", "lg_device.cuh", "lg_kernels.cuh", "lg_capi.cuh", "lg_prefill.cuh", "lg_attn_deep.cuh", "lg_attn_cluster.cuh"],
            "lg_plan.cu": ["lg_engine.h", "lg_device.cuh", "lg_dense.cuh", "lg_latent.cuh", "lg_seq.cuh", "lg_ssd.cuh", "lg_window.cuh", "lg_plan_seq.cuh"]}
HEADERS = [os.path.join(INC, f) for f in ("lg_abi.h", "lg_b200.h", "lg_plan.h")] + [os.path.join(HOST, f) for f in ("lg_host.h", "lg_formats.h")]
SELF = os.path.abspath(__file__)


def sources(f: str) -> list[str]:
    """Everything an object file depends on."""
    if f in CUDA_SRC:
        return [os.path.join(CUDA, g) for g in [f] + CUDA_SRC[f]] + HEADERS + [SELF]
    return [os.path.join(HOST, f)] + HEADERS + [SELF]


def newer(deps: list[str], target: str) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def stale() -> bool:
    return any(newer(sources(f), LIB) for f in [*HOST_SRC, *CUDA_SRC])


def build(mtp_n: int = 4, force: bool = False, ptxas_v: bool = False, stamps: bool = False) -> str:
    if not force and not stale():
        return LIB
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    defs = [f"-DLG_MTP_N={mtp_n}"] + (["-DLG_STAMPS"] if stamps else [])     # stamps: profiling build with phase time stamps
    # objects are reused only between builds with the same options
    tag = os.path.join(objdir, "options")
    want = " ".join(defs)
    same = os.path.exists(tag) and open(tag).read() == want
    jobs, objs = [], []
    for f in [*CUDA_SRC, *HOST_SRC]:                                          # the CUDA units first: they take longest
        o = os.path.join(objdir, f + ".o")
        objs.append(o)
        if same and not force and not newer(sources(f), o):
            continue
        if f in CUDA_SRC:
            cmd = [NVCC, "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
                   "-Xcompiler", "-fPIC", *defs, f"-I{INC}", f"-I{HOST}", f"-I{CUDA}", "-c", os.path.join(CUDA, f), "-o", o]
            if ptxas_v:
                cmd[1:1] = ["-Xptxas", "-v"]
        else:
            cmd = ["gcc", "-O2", "-fPIC", "-std=gnu11", "-Wall", "-Wextra", *defs, f"-I{INC}", f"-I{HOST}",
                   "-c", os.path.join(HOST, f), "-o", o]
        jobs.append((cmd, subprocess.Popen(cmd)))
    failed = [cmd for cmd, p in jobs if p.wait() != 0]
    if failed:
        raise subprocess.CalledProcessError(1, failed[0])
    with open(tag, "w") as t:
        t.write(want)
    tmp = f"{LIB}.{os.getpid()}"                                              # a reader never sees half a library
    subprocess.check_call([NVCC, "-shared", "-o", tmp, *objs, "-lcudart"])
    os.replace(tmp, LIB)
    return LIB


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--mtp-n", type=int, default=4)
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--ptxas-v", action="store_true")
    ap.add_argument("--stamps", action="store_true", help="profiling build: kernels record phase time stamps (lg_debug_stamps)")
    a = ap.parse_args()
    print(build(a.mtp_n, a.force or a.stamps, a.ptxas_v, a.stamps))
