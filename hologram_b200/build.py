"""Build libhologram_b200.so (sm_100a only) in-tree with nvcc.

Run: python hologram_b200/build.py [--force] [--verbose] [--serving]   (by path: importing the package needs the built library)

`--serving` builds libhologram_b200_serving.so instead: the archive session and the kernels a decoder model served from a
checkpoint uses, without the other families (calls that need those are refused). The package loads it only where the full
library has not been built.
"""
import os
import re
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libhologram_b200.so")
SOURCES = ["api.cu", "lut.cu", "glue.cu", "attention.cu", "gemm.cu", "linear.cu", "causal_attention.cu", "window_attention.cu", "retention.cu", "moe.cu", "quant_gemv.cu", "tp.cu", "session.cu", "addressed.cpp", "pool.cpp", "archive.cpp", "blake3.cpp", "label.cpp"]
SERVING_LIB = os.path.join(HERE, "libhologram_b200_serving.so")
SERVING_SOURCES = ["api.cu", "glue.cu", "linear.cu", "causal_attention.cu", "window_attention.cu", "retention.cu", "moe.cu", "session.cu", "addressed.cpp", "pool.cpp", "archive.cpp", "blake3.cpp", "label.cpp",
                   "absent_families.cpp"]
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fno-fast-math", "--expt-relaxed-constexpr",
]


def _nvcc():
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    return "nvcc"


def _deps(src):
    """`src` and the headers it includes, directly or through other headers."""
    deps, todo = [], [src]
    while todo:
        path = todo.pop()
        if path in deps or not os.path.exists(path):
            continue
        deps.append(path)
        with open(path, encoding="utf-8") as f:
            names = re.findall(r'^#include "([^"]+)"', f.read(), re.M)
        todo += [os.path.normpath(os.path.join(os.path.dirname(path), n)) for n in names]
    return deps


def build_for_serving():
    """What serving a checkpoint needs: the full library where it exists (brought up to date), else the serving build."""
    return build() if os.path.exists(LIB) else build(serving=True)


def build(force=False, verbose=False, serving=False):
    lib, sources = (SERVING_LIB, SERVING_SOURCES) if serving else (LIB, SOURCES)
    objs = []
    procs = []
    for name in sources:
        src = os.path.join(CSRC, name)
        obj = os.path.join(CSRC, os.path.splitext(name)[0] + ".o")
        objs.append(obj)
        newest = max(os.path.getmtime(d) for d in _deps(src))
        if force or not os.path.exists(obj) or os.path.getmtime(obj) < newest:
            cmd = [_nvcc()] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", src, "-o", obj]
            procs.append((name, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for name, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0 or verbose:
            sys.stderr.write(f"--- {name} ---\n{out}\n")
        failed |= p.returncode != 0
    if failed:
        raise RuntimeError("nvcc failed")
    if force or procs or not os.path.exists(lib) or os.path.getmtime(lib) < max(os.path.getmtime(o) for o in objs):
        cmd = [_nvcc(), "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", lib] + objs + ["-ldl"]
        subprocess.check_call(cmd)
    return lib


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, serving="--serving" in sys.argv))
