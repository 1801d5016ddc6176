"""Builds libornith_cuda.so in-tree with nvcc for sm_100a.

Run as `python ornith-rs_b200/build.py` or through `__graft_entry__.build()`.
Objects are rebuilt only when a source or header is newer.  `-fmad=false`
and `-ffp-contract=off` are part of the numerical contract: a fused
multiply-add happens only where the source writes `fmaf`.
"""
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB = os.path.join(HERE, "libornith_cuda.so")
SOURCES = ["api.cu", "linear.cu", "ops.cu", "gdn.cu", "attn.cu", "sample.cu", "model.cu", "loader.cu", "fused.cu", "gemm.cu", "ep.cu", "batch.cu", "flash.cu", "gdn_chunk.cu",
           "decoder.cu", "dense.cu", "latent.cu", "heads.cu", "decayed.cu", "grouped.cu"]
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-fmad=false", "-Xcompiler", "-fPIC,-ffp-contract=off,-fno-fast-math", "-Xptxas", "-v",
]


def _newest_header():
    t = 0.0
    for root in (CSRC, os.path.join(HERE, "..", "include")):
        for f in os.listdir(root):
            if f.endswith((".h", ".cuh")):
                t = max(t, os.path.getmtime(os.path.join(root, f)))
    return t


def _compile(src, verbose):
    obj = os.path.join(OBJ, src.replace(".cu", ".o"))
    spath = os.path.join(CSRC, src)
    if os.path.exists(obj) and os.path.getmtime(obj) > max(os.path.getmtime(spath), _newest_header()):
        return obj, ""
    cmd = [NVCC] + FLAGS + ["-c", spath, "-o", obj]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("nvcc failed for %s:\n%s\n%s" % (src, r.stdout, r.stderr))
    return obj, r.stderr


def _up_to_date():
    """The library is newer than everything it is made from (it may have travelled without its objects)."""
    if not os.path.exists(LIB):
        return False
    newest = max([os.path.getmtime(os.path.join(CSRC, s)) for s in SOURCES] + [os.path.getmtime(os.path.abspath(__file__)), _newest_header()])
    return os.path.getmtime(LIB) > newest


def build(verbose=False):
    if _up_to_date():
        return LIB
    os.makedirs(OBJ, exist_ok=True)
    with ThreadPoolExecutor(max_workers=8) as ex:
        results = list(ex.map(lambda s: _compile(s, verbose), SOURCES))
    objs = [o for o, _ in results]
    log = "".join(l for _, l in results)
    if log:
        with open(os.path.join(OBJ, "ptxas.log"), "a") as f:
            f.write(log)
    if not _up_to_date():
        cmd = [NVCC, "-shared", "-o", LIB] + objs + ["-lcudart", "-ldl"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("link failed:\n%s\n%s" % (r.stdout, r.stderr))
    if verbose:
        sys.stdout.write(log)
    return LIB


if __name__ == "__main__":
    print(build(verbose="-v" in sys.argv))
