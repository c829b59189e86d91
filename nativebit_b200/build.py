"""In-tree build of the kernel libraries (hand-written CUDA for sm_100a, C ABI).

    python -m nativebit_b200.build          # or nativebit_b200.build.build_library()

Two libraries share their sources' objects: libnativebit_b200.so (packed models, include/nativebit_b200.h) and
libnativebit_b200_layered.so (layered models, include/nativebit_b200_layered.h), so that a program which serves one
kind of model compiles only what that kind needs.  nvcc cross-compiles without a GPU.  The libraries are written
next to this file so that they travel with the source tree; nothing is installed into site-packages.
"""
from __future__ import annotations

import fcntl
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB_NAME = "libnativebit_b200.so"
LAYERED_LIB_NAME = "libnativebit_b200_layered.so"
LIB_PATH = os.path.join(HERE, LIB_NAME)
ARCH_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a"]


def _nvcc() -> str:
    cand = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(cand):
        raise RuntimeError("nvcc not found; the CUDA toolkit is required to build nativebit_b200")
    return cand


# library -> its sources under csrc/
LIBRARIES = {
    "packed": (LIB_NAME, ("nb_host", "nb_unpack", "nb_gemm", "nb_gemm_fused", "nb_gemv", "nb_stream", "nb_decode", "nb_comm")),
    "layered": (LAYERED_LIB_NAME, ("nb_host", "nb_unpack", "nb_gemm", "nb_decode", "nb_linear", "nb_latent", "nb_gla", "nb_talk")),
}


def library_path(which: str = "packed") -> str:
    return os.path.join(HERE, LIBRARIES[which][0])


def _inputs(src: str) -> list[str]:
    """Files an object depends on: its source, every header, this script."""
    heads = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    inc = os.path.join(HERE, "..", "include")
    heads += [os.path.join(inc, f) for f in os.listdir(inc)]
    return [src, os.path.abspath(__file__), *heads]


def _older(path: str, inputs: list[str]) -> bool:
    if not os.path.exists(path):
        return True
    t = os.path.getmtime(path)
    return any(os.path.getmtime(d) > t for d in inputs)


def is_stale(which: str = "packed") -> bool:
    """True if the library is missing or older than one of its sources."""
    deps = [d for stem in LIBRARIES[which][1] for d in _inputs(os.path.join(CSRC, stem + ".cu"))]
    return _older(library_path(which), deps)


def build_library(force: bool = False, verbose: bool = False, which: str = "packed") -> str:
    """Compile one library's sources (only those whose object is out of date) and link it; returns its path."""
    path = library_path(which)
    if not force and not is_stale(which):
        return path
    obj_dir = os.path.join(HERE, "build")
    os.makedirs(obj_dir, exist_ok=True)
    with open(os.path.join(obj_dir, "lock"), "w") as lock:      # two processes never write the same object
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and not is_stale(which):
            return path
        nvcc = _nvcc()
        common = ARCH_FLAGS + ["-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC"]
        if verbose:
            common += ["-Xptxas", "-v"]
        procs, objs = [], []
        for stem in LIBRARIES[which][1]:
            src, obj = os.path.join(CSRC, stem + ".cu"), os.path.join(obj_dir, stem + ".o")
            objs.append(obj)
            if force or _older(obj, _inputs(src)):
                procs.append((src, obj, subprocess.Popen([nvcc, *common, "-c", src, "-o", obj + ".tmp"],
                                                         stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
        failed = None
        for src, obj, p in procs:
            out, _ = p.communicate()
            if verbose or p.returncode:
                sys.stderr.write(out)
            if p.returncode:
                failed = failed or src
            else:
                os.replace(obj + ".tmp", obj)
        if failed:
            raise RuntimeError(f"nvcc failed on {failed}")
        tmp = path + ".tmp"
        r = subprocess.run([nvcc, *ARCH_FLAGS, "-shared", "-o", tmp, *objs], stdout=subprocess.PIPE,
                           stderr=subprocess.STDOUT, text=True)
        if r.returncode:
            sys.stderr.write(r.stdout)
            raise RuntimeError("link failed")
        os.replace(tmp, path)
    return path


def build_all(force: bool = False, verbose: bool = False) -> list[str]:
    return [build_library(force, verbose, which) for which in LIBRARIES]


if __name__ == "__main__":
    print(*build_all(force="--force" in sys.argv, verbose="-v" in sys.argv), sep="\n")
