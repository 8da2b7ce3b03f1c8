"""Builds the CUDA libraries for sm_100a with nvcc, in-tree, beside this file.

    python zk-deepseek_b200/build.py [--force] [--verbose] [NAME ...]

    libint64gemm.so   the int64 fixed-point kernels of the integer model
    libfloatops.so    the kernels of the floating-point decoder designs

nvcc cross-compiles without a GPU.  The libraries link the CUDA runtime statically and resolve the driver entry
points they need (tensor-map encoding) at run time, so they load on a machine without a GPU as well.  A library is
compiled when it is missing or older than one of its sources; callers on a fresh checkout build only the one they
load.
"""
import fcntl
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
INCLUDE = os.path.join(os.path.dirname(HERE), "include")
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
         "-Xcompiler", "-fPIC"]
# library -> (translation units, headers)
LIBRARIES = {
    "libint64gemm.so": (["capi.cu", "fixedpoint.cu", "gemm_exact.cu", "limb_gemm.cu", "converters.cu"],
                        ["common.cuh", "kernels.h", "tcgen05.cuh", "zkds_int64.h"]),
    "libfloatops.so": (["float_capi.cu", "float_ops.cu", "float_gemm.cu", "float_gemm_tc.cu", "float_attention.cu",
                        "float_grouped.cu", "float_recurrent.cu", "float_scan_tc.cu"],
                       ["common.cuh", "float_common.cuh", "tcgen05.cuh", "zkds_float.h"]),
}
INT_LIBRARY, FLOAT_LIBRARY = "libint64gemm.so", "libfloatops.so"
OUT = os.path.join(HERE, INT_LIBRARY)


def _dep(name):
    path = os.path.join(CSRC, name)
    return path if os.path.exists(path) else os.path.join(INCLUDE, name)


def _stale(library):
    out = os.path.join(HERE, library)
    if not os.path.exists(out):
        return True
    t = os.path.getmtime(out)
    sources, headers = LIBRARIES[library]
    return any(os.path.getmtime(_dep(d)) > t for d in sources + headers)


def _compile(library, verbose):
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    out = os.path.join(HERE, library)
    tag = ".%d.partial" % os.getpid()
    flags = FLAGS + (["-Xptxas", "-v"] if verbose else [])
    objs, jobs, failed = [], [], False
    for src in LIBRARIES[library][0]:                  # the translation units compile side by side
        obj = os.path.join(HERE, src + tag + ".o")
        objs.append(obj)
        jobs.append(subprocess.Popen([nvcc] + flags + ["-x", "cu", "-c", os.path.join(CSRC, src), "-o", obj],
                                     stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True))
    for job in jobs:
        text = job.communicate()[0]
        if verbose or job.returncode:
            sys.stderr.write(text)
        failed |= job.returncode != 0
    try:
        if not failed:
            # the library appears under its name only once it is complete
            res = subprocess.run([nvcc] + FLAGS[:2] + ["-shared", "-Xcompiler", "-fPIC", "-o", out + tag] + objs,
                                 capture_output=True, text=True)
            failed = res.returncode != 0
            if failed:
                sys.stderr.write(res.stdout + res.stderr)
        if failed:
            raise RuntimeError("nvcc failed building " + library)
        os.replace(out + tag, out)
    finally:
        for f in objs + [out + tag]:
            if os.path.exists(f):
                os.remove(f)
    return out


def build(force=False, verbose=False, library=INT_LIBRARY):
    out = os.path.join(HERE, library)
    if not force and not _stale(library):
        return out
    with open(out + ".lock.partial", "w") as lock:     # one process compiles, the others wait for it
        fcntl.flock(lock, fcntl.LOCK_EX)
        if force or _stale(library):
            _compile(library, verbose)
    return out


if __name__ == "__main__":
    names = [a for a in sys.argv[1:] if not a.startswith("-")] or list(LIBRARIES)
    for name in names:
        print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, library=name))
