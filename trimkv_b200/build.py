"""Builds libtrimkv_b200.so in-tree with nvcc for sm_100a (cross-compiles without a GPU)."""
from __future__ import annotations

import os
import shutil
import subprocess

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libtrimkv_b200.so")
SOURCES = ["tkv_abi.cu", "tkv_append.cu", "tkv_evict.cu", "tkv_attn.cu", "tkv_attn_tc.cu", "tkv_attn_multi.cu", "tkv_attn_prefill.cu", "tkv_gemm_tc.cu", "tkv_fused.cu",
           "tkv_stream.cu", "tkv_linrec.cu", "tkv_linrec_chunk.cu", "tkv_linrec_tc.cu", "tkv_diffattn.cu", "tkv_diffattn_tc.cu",
           "tkv_chanrec.cu", "tkv_chanrec_chunk.cu", "tkv_chanrec_tc.cu", "tkv_latent.cu", "tkv_latent_tc.cu", "tkv_moe.cu", "tkv_moe_tc.cu"]
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "--use_fast_math=false",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found; set NVCC or install the CUDA toolkit")


def needs_build() -> bool:
    if not os.path.exists(LIB):
        return True
    t = os.path.getmtime(LIB)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC)] + [
        os.path.join(HERE, "..", "include", "trimkv_b200.h"), os.path.abspath(__file__)]
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False) -> str:
    """Compile every .cu under csrc/ into one shared library; returns its path."""
    if not force and not needs_build():
        return LIB
    nvcc = _nvcc()
    flags = [f for f in NVCC_FLAGS if not f.startswith("--use_fast_math")]
    if verbose:
        flags += ["-Xptxas", "-v"]
    objs = [os.path.join(CSRC, src.replace(".cu", ".o")) for src in SOURCES]
    cmds = [[nvcc, *flags, "-c", os.path.join(CSRC, src), "-o", obj] for src, obj in zip(SOURCES, objs)]
    procs = [subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True) for cmd in cmds]
    failed = []
    for src, cmd, proc in zip(SOURCES, cmds, procs):       # the translation units are independent: compile them side by side
        out, err = proc.communicate()
        if verbose or proc.returncode != 0:
            print(" ".join(cmd)); print(out); print(err)
        if proc.returncode != 0:
            failed.append(src)
    if failed:
        raise RuntimeError(f"nvcc failed on {', '.join(failed)}")
    cmd = [nvcc, "-shared", "-o", LIB, *objs, "-gencode", "arch=compute_100a,code=sm_100a"]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        print(r.stdout); print(r.stderr)
        raise RuntimeError("link failed")
    return LIB


if __name__ == "__main__":
    import sys
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
