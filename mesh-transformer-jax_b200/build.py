"""Builds libmtj_b200.so (sm_100a) in-tree with nvcc.

Usage: python build.py [--force] [--verbose] [--family stack]

``--family stack`` compiles only the units that layer-stack models use, into libmtj_b200_stack.so: what a program that
serves one such model needs on its first call.
"""
from __future__ import annotations

import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "libmtj_b200.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
         "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr"]
# the units of one family's library; None: all of them
FAMILIES = {
    None: None,
    "stack": ("mtj_model", "mtj_stack", "mtj_stack_kernels", "mtj_latent_attn", "mtj_attn_tc_latent", "mtj_ssm", "mtj_gemm_tc",
              "mtj_gemm_tc_stack", "mtj_gemm_tc_stack_post", "mtj_grouped_attn", "mtj_attn_tc_grouped", "mtj_matrix_state", "mtj_matrix_chunk", "mtj_gemv", "mtj_misc", "mtj_sample", "mtj_loss", "mtj_family_stubs"),
}


def library(family=None) -> str:
    return OUT if family is None else os.path.join(HERE, f"libmtj_b200_{family}.so")


def sources(family=None):
    units = FAMILIES[family]
    names = sorted(f for f in os.listdir(CSRC) if f.endswith(".cu"))
    return [os.path.join(CSRC, f) for f in names if units is None or f[:-3] in units]


def stale(family=None) -> bool:
    out = library(family)
    if not os.path.exists(out):
        return True
    t = os.path.getmtime(out)
    deps = sources(family) + [os.path.join(CSRC, f) for f in os.listdir(CSRC) if not f.endswith(".cu")]
    deps.append(os.path.join(HERE, "..", "include", "mtj_b200.h"))
    return any(os.path.getmtime(d) > t for d in deps)


def ensure(family) -> str:
    """A library that serves ``family``: the whole one if it is built and current, else the family's own."""
    return OUT if not stale() else build(family=family)


def build(force: bool = False, verbose: bool = False, family=None) -> str:
    out_path = library(family)
    if not force and not stale(family):
        return out_path
    objs = []
    procs = []
    os.makedirs(os.path.join(HERE, "build"), exist_ok=True)
    units = [(src, "", []) for src in sources(family)]
    if family is None:
        # the whole-step decode kernel a second time with one 512-thread block per SM (see the head of that file)
        units.append((os.path.join(CSRC, "mtj_decode_mega.cu"), "_mt512", ["-DMTJ_MEGA_MT=512"]))
    for src, tag, extra in units:
        obj = os.path.join(HERE, "build", os.path.basename(src)[:-3] + tag + ".o")
        cmd = [NVCC, *FLAGS, *extra, "-c", src, "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
        objs.append(obj)
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        if out.strip() and (verbose or p.returncode):
            print(out)
        if p.returncode:
            print(f"nvcc failed on {src}", file=sys.stderr)
            failed = True
    if failed:
        raise RuntimeError("nvcc failed")
    tmp = out_path + f".{os.getpid()}"
    subprocess.check_call([NVCC, "-shared", "-o", tmp, *objs, "-lcudart"])
    os.replace(tmp, out_path)
    return out_path


if __name__ == "__main__":
    fam = sys.argv[sys.argv.index("--family") + 1] if "--family" in sys.argv else None
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, family=fam))
