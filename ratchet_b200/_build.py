"""In-tree build of ``libratchet_cuda.so`` (sm_100a only) with nvcc.

Every ``csrc/*.cu`` file is compiled to an object in ``csrc/_obj/`` (parallel, skipped when the
object is newer than its sources) and linked into ``ratchet_b200/libratchet_cuda.so``.  nvcc
cross-compiles without a GPU, so this runs on a CPU-only machine as well.
"""
from __future__ import annotations

import concurrent.futures as cf
import glob
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(CSRC, "_obj")
LIB = os.path.join(HERE, "libratchet_cuda.so")
CORE_LIB = os.path.join(HERE, "libratchet_cuda_core.so")
NOT_CORE = {"decode.cu", "comm.cu", "gguf.cu"}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]


def nvcc() -> str:
    path = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(path):
        raise RuntimeError("nvcc not found: the CUDA library cannot be built")
    return path


def _headers():
    return glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h")) + \
        glob.glob(os.path.join(HERE, "..", "include", "*.h"))


def _stale(target: str, sources) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(s) > t for s in sources)


def _compile(src: str, verbose: bool) -> str:
    obj = os.path.join(OBJ, os.path.basename(src)[:-3] + ".o")
    if _stale(obj, [src] + _headers()):
        cmd = [nvcc()] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", src, "-o", obj]
        proc = subprocess.run(cmd, capture_output=True, text=True)
        if proc.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src}:\n{proc.stdout}\n{proc.stderr}")
        if verbose:
            sys.stderr.write(proc.stderr)
    return obj


def build(force: bool = False, verbose: bool = False) -> str:
    os.makedirs(OBJ, exist_ok=True)
    if force:
        for f in glob.glob(os.path.join(OBJ, "*.o")):
            os.remove(f)
    return _link(LIB, _sources(), verbose)


def _sources(core: bool = False):
    return [s for s in sorted(glob.glob(os.path.join(CSRC, "*.cu"))) if not (core and os.path.basename(s) in NOT_CORE)]


def _link(lib: str, sources, verbose: bool) -> str:
    # the longest translation units first: they decide how long a parallel build takes
    by_size = sorted(sources, key=os.path.getsize, reverse=True)
    with cf.ThreadPoolExecutor(max_workers=min(len(sources), max(8, os.cpu_count() or 8))) as ex:
        objs = sorted(ex.map(lambda s: _compile(s, verbose), by_size))
    if _stale(lib, objs):
        part = f"{lib}.{os.getpid()}"
        cmd = [nvcc(), "-shared", "-o", part] + objs + ["-gencode", "arch=compute_100a,code=sm_100a", "-lcudart", "-ldl"]
        proc = subprocess.run(cmd, capture_output=True, text=True)
        if proc.returncode != 0:
            raise RuntimeError(f"link failed:\n{proc.stdout}\n{proc.stderr}")
        os.replace(part, lib)
    return lib


def ensure_runtime() -> str:
    """Path of a library that is newer than its sources: the full one where it has been built, else the core library,
    built first if need be."""
    if not _stale(LIB, _sources() + _headers()):
        return LIB
    if _stale(CORE_LIB, _sources(core=True) + _headers()):
        os.makedirs(OBJ, exist_ok=True)
        _link(CORE_LIB, _sources(core=True), False)
    return CORE_LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
