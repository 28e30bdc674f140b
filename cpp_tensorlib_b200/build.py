"""Compile the CUDA sources of this package into ``libtlb200.so`` (sm_100a only).

Usage: ``python -m cpp_tensorlib_b200.build [--force] [--verbose]``.  The shared
object is written next to this file so it travels with the source tree; it
links the CUDA runtime statically and nothing else.
"""
import glob
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libtlb200.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-lineinfo", "-std=c++17",
         "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr", "-cudart", "static"]


def sources():
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")))


def _headers():
    return glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(HERE, "..", "include", "*.h"))


def _newer(target, deps):
    return os.path.exists(target) and all(os.path.getmtime(d) <= os.path.getmtime(target) for d in deps)


def _stale():
    return not _newer(LIB, sources() + _headers())


def _includes(path, seen):
    """The project headers a source reaches through its quoted includes."""
    with open(path) as f:
        for line in f:
            if line.startswith('#include "'):
                h = os.path.normpath(os.path.join(os.path.dirname(path), line.split('"')[1]))
                if h not in seen and os.path.exists(h):
                    seen.add(h)
                    _includes(h, seen)
    return seen


def build(force=False, verbose=False):
    if not (force or _stale()):
        return LIB
    objs = []
    procs = []
    for src in sources():
        obj = src[:-3] + ".o"
        objs.append(obj)
        if not (force or verbose) and _newer(obj, [src] + sorted(_includes(src, set()))):
            continue
        cmd = [NVCC] + FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", src, "-o", obj]
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT)))
    for src, p in procs:
        out, _ = p.communicate()
        if verbose or p.returncode:
            sys.stderr.write(out.decode())
        if p.returncode:
            raise RuntimeError("nvcc failed on " + src)
    subprocess.check_call([NVCC, "-shared", "-cudart", "static", "-o", LIB] + objs +
                          ["-Xcompiler", "-fPIC"])
    return LIB


if __name__ == "__main__":
    print(build("--force" in sys.argv, "--verbose" in sys.argv))
