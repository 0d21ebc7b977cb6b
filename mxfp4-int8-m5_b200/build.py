"""Builds the C-ABI libraries in-tree with nvcc for sm_100a: libscmx.so (the W4A8 path) and libscmx_mixers.so (sequence mixers
of the hybrid decoder models).  A caller builds only the library it needs.

Usage: python build.py [--force] [--verbose] [--only scmx|mixers]
"""
import os
import subprocess
import sys
import tempfile

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
INCLUDE = os.path.join(HERE, "..", "include")
LIBS = {"scmx": os.path.join(HERE, "libscmx.so"), "mixers": os.path.join(HERE, "libscmx_mixers.so")}
LIB = LIBS["scmx"]
SHARED = ("scmx_abi.cu", "scmx_tma.cu")        # error reporting and tensor maps: part of both libraries
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-lineinfo", "-std=c++17", "-Xcompiler", "-fPIC",
              "--shared", "-cudart", "static"]


def sources(which="scmx"):
    d = CSRC if which == "scmx" else os.path.join(CSRC, "mixers")
    own = [os.path.join(d, f) for f in os.listdir(d) if f.endswith(".cu")]
    return sorted(own if which == "scmx" else own + [os.path.join(CSRC, f) for f in SHARED])


def _deps(which):
    dirs = [CSRC, INCLUDE] + ([os.path.join(CSRC, "mixers")] if which == "mixers" else [])
    files = [os.path.join(d, f) for d in dirs for f in os.listdir(d) if f.endswith((".cuh", ".h"))]
    return files + sources(which)


def _stale(which="scmx"):
    if not os.path.exists(LIBS[which]):
        return True
    t = os.path.getmtime(LIBS[which])
    return any(os.path.getmtime(d) > t for d in _deps(which))


def _nvcc():
    if "NVCC" in os.environ:
        return os.environ["NVCC"]
    cuda = os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "bin", "nvcc")
    return cuda if os.path.exists(cuda) else "nvcc"


def build(force=False, verbose=False, which="scmx"):
    """Compile the sources of one library when it is missing or older than a source; returns the library path."""
    if not force and not _stale(which):
        return LIBS[which]
    nvcc = _nvcc()
    objs = []
    procs = []
    os.makedirs(os.path.join(HERE, "build"), exist_ok=True)
    work = tempfile.mkdtemp(dir=os.path.join(HERE, "build"))
    for src in sources(which):
        obj = os.path.join(work, os.path.basename(src)[:-3] + ".o")
        objs.append(obj)
        cmd = [nvcc, *[f for f in NVCC_FLAGS if f != "--shared"], "-c", src, "-o", obj] + (["-Xptxas", "-v"] if verbose else [])
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = []
    for src, p in procs:
        out, _ = p.communicate()
        if verbose or p.returncode:
            sys.stderr.write(out)
        if p.returncode:
            failed.append(src)
    if failed:
        raise RuntimeError(f"nvcc failed on {', '.join(failed)}")
    tmp = os.path.join(work, os.path.basename(LIBS[which]))
    subprocess.run([nvcc, *NVCC_FLAGS, *objs, "-o", tmp], check=True)
    os.replace(tmp, LIBS[which])
    for o in objs:
        os.unlink(o)
    os.rmdir(work)
    return LIBS[which]


if __name__ == "__main__":
    only = sys.argv[sys.argv.index("--only") + 1] if "--only" in sys.argv else None
    for name in LIBS:
        if only in (None, name):
            print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, which=name))
