"""In-tree build of the CUDA libraries with nvcc for sm_100a (cross-compiles without a GPU).

``libglorcq_b200.so`` serves the quantized decoders, ``libglorcq_b200_dense.so`` the unquantized ones; each is
compiled only when something asks for it.  Every source is an object of its own (compiled side by side), and a
library appears under its name only when it is complete, so that processes that start together never load half a file.
"""

from __future__ import annotations

import fcntl
import os
import subprocess
import tempfile
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
INCLUDE = os.path.join(HERE, "..", "include")
LIB = os.path.join(HERE, "libglorcq_b200.so")
DENSE_LIB = os.path.join(HERE, "libglorcq_b200_dense.so")
SOURCES = {LIB: ["api.cu", "moe.cu", "attn.cu", "lm_head.cu"],
           DENSE_LIB: ["dense_mm.cu", "dense_aux.cu", "dense_head.cu", "mlstm.cu", "decay_attn.cu", "gqa_attn.cu", "latent_attn.cu"]}
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC"]


def _stale(lib: str) -> bool:
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cuh")]
    deps += [os.path.join(CSRC, f) for f in SOURCES[lib]] + [os.path.join(INCLUDE, f) for f in os.listdir(INCLUDE)]
    return any(os.path.getmtime(d) > t for d in deps)


def _run(cmd, verbose):
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError("nvcc failed:\n" + " ".join(cmd) + "\n" + res.stdout + res.stderr)
    if verbose:
        print(res.stderr)


def build(force: bool = False, verbose: bool = False, lib: str = LIB) -> str:
    """Compile the sources of ``lib`` into glorcq_b200/; returns the library path."""
    if not force and not _stale(lib):
        return lib
    nvcc = os.environ.get("NVCC", "nvcc")
    with open(lib + ".lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not force and not _stale(lib):        # another process built it meanwhile
            return lib
        with tempfile.TemporaryDirectory(dir=HERE, prefix=".build-") as tmp:
            objs = [os.path.join(tmp, s[:-3] + ".o") for s in SOURCES[lib]]
            cmds = [[nvcc] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", os.path.join(CSRC, s), "-o", o]
                    for s, o in zip(SOURCES[lib], objs)]
            with ThreadPoolExecutor(max(1, min(len(cmds), os.cpu_count() or 1))) as ex:
                list(ex.map(lambda c: _run(c, verbose), cmds))
            part = os.path.join(tmp, "lib.so")
            _run([nvcc] + NVCC_FLAGS + ["-shared", "-o", part] + objs, verbose)
            os.replace(part, lib)
    return lib


def build_all(force: bool = False, verbose: bool = False):
    return [build(force, verbose, lib) for lib in SOURCES]


if __name__ == "__main__":
    import sys
    print(build_all(force=True, verbose="-v" in sys.argv))
