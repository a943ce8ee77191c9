"""In-tree build of ``librunit_cuda.so`` (hand-written CUDA for sm_100a, C ABI in include/runit_cuda.h).

``python -m runit_mac_b200.build`` compiles every ``csrc/*.cu`` with nvcc for
``arch=compute_100a,code=sm_100a`` and links one shared library beside this file.  nvcc
cross-compiles without a GPU.  Objects are rebuilt only when a source or header is newer.
"""
from __future__ import annotations

import fcntl
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
INCLUDE = PKG.parent / "include"
OBJ = PKG / "build"
LIB = PKG / "librunit_cuda.so"

# Parts of the library that are useful alone: {name: (shared library, sources)}.  A part exports the subset of the C ABI its
# sources define; it exists so that serving one kind of model does not compile the kernels of all others.
PARTS = {
    "layered": (PKG / "librunit_layered.so",
                ("ctx", "gemv_stream", "model_core", "layered_model", "gemv_bf16", "gemm_bf16", "latent_attention", "head_attention", "linear_state", "moe_route",
                 "moe_permute", "sampler")),
}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xptxas", "-v" if os.environ.get("RUNIT_PTXAS_V") else "-O3",
    "-Xcompiler", "-fPIC,-O2,-Wall", "-I", str(INCLUDE), "-I", str(CSRC),
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found; the CUDA toolkit is required to build librunit_cuda.so")


def _newest_header() -> float:
    hs = list(CSRC.glob("*.h")) + list(CSRC.glob("*.cuh")) + list(INCLUDE.glob("*.h")) + [Path(__file__)]
    return max(h.stat().st_mtime for h in hs)


def _fresh(lib: Path, srcs) -> bool:
    """The library exists and is newer than everything it is made from."""
    return lib.exists() and lib.stat().st_mtime >= max([_newest_header()] + [s.stat().st_mtime for s in srcs])


def ensure(part: str) -> Path:
    """A library that holds `part`: the full one when it is built and current, else the part's own, compiled on demand."""
    if _fresh(LIB, CSRC.glob("*.cu")):
        return LIB
    lib, names = PARTS[part]
    if not _fresh(lib, [CSRC / (n + ".cu") for n in names]):
        OBJ.mkdir(exist_ok=True)
        with open(OBJ / ".lock", "w") as lock:      # one builder at a time
            fcntl.flock(lock, fcntl.LOCK_EX)
            build(part=part)
    return lib


def build(force: bool = False, verbose: bool = False, part: str | None = None) -> Path:
    nvcc = _nvcc()
    OBJ.mkdir(exist_ok=True)
    hdr = _newest_header()
    out, names = PARTS[part] if part else (LIB, None)
    srcs = [CSRC / (n + ".cu") for n in names] if names else sorted(CSRC.glob("*.cu"))
    todo = []
    for s in srcs:
        o = OBJ / (s.stem + ".o")
        if force or not o.exists() or o.stat().st_mtime < max(s.stat().st_mtime, hdr):
            todo.append((s, o))

    def compile_one(so):
        s, o = so
        cmd = [nvcc, *NVCC_FLAGS, "-c", str(s), "-o", str(o)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("nvcc failed for %s:\n%s\n%s" % (s.name, r.stdout, r.stderr))
        if verbose or os.environ.get("RUNIT_PTXAS_V"):
            sys.stderr.write(r.stderr)
        return o

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(todo)))) as ex:
        list(ex.map(compile_one, todo))
    objs = [OBJ / (s.stem + ".o") for s in srcs]
    if todo or not out.exists() or out.stat().st_mtime < max(o.stat().st_mtime for o in objs):
        tmp = out.with_name("%s.%d.tmp" % (out.name, os.getpid()))
        cmd = [nvcc, "-shared", "-Xlinker", "-z,defs", "-o", str(tmp), *map(str, objs), "-lcudart"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("link failed:\n%s\n%s" % (r.stdout, r.stderr))
        os.replace(tmp, out)
    return out


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
