"""Build the C-ABI CUDA libraries in-tree with nvcc for sm_100a.

    python -m mini_sgl_integer_b200.build [int] [float] [--force] [--verbose]

``libb200int.so`` holds the integer path, ``libb200float.so`` the floating-point models; a model needs only its own.
nvcc cross-compiles without a GPU, so this runs on a CPU-only host as well.
"""
from __future__ import annotations

import fcntl
import os
import shutil
import subprocess
import sys

PKG_DIR = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG_DIR, "csrc")
INCLUDE = os.path.join(os.path.dirname(PKG_DIR), "include")
LIBRARIES = {
    "int": ("libb200int.so", ["runtime.cu", "api.cu", "batch_ops.cu", "rowops.cu", "attn.cu", "attn_split.cu", "attn_prefill.cu",
                              "gemm.cu", "model_ops.cu", "tp.cu"]),
    "float": ("libb200float.so", ["runtime.cu", "batch_ops.cu", "float_gemm.cu", "float_rows.cu", "recurrent.cu", "latent_attn.cu", "matrix_memory.cu",
                                  "grouped_attn.cu"]),
}
LIB_PATH = os.path.join(PKG_DIR, LIBRARIES["int"][0])
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found (set NVCC or put it on PATH)")


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def library_path(which: str = "int") -> str:
    return os.path.join(PKG_DIR, LIBRARIES[which][0])


def build_library(force: bool = False, verbose: bool = False, which: str = "int") -> str:
    """Compile the sources of one library (``which`` of LIBRARIES) and link them; returns its path.  Processes that build
    at the same time wait for each other."""
    obj_dir = os.path.join(PKG_DIR, "build")
    os.makedirs(obj_dir, exist_ok=True)
    with open(os.path.join(obj_dir, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build_locked(obj_dir, force, verbose, which)


def _build_locked(obj_dir: str, force: bool, verbose: bool, which: str) -> str:
    target, sources = library_path(which), LIBRARIES[which][1]
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".inc", ".h"))]
    headers += [os.path.join(INCLUDE, f) for f in os.listdir(INCLUDE) if f.endswith(".h")]
    objs, procs, nvcc = [], [], None
    for src in sources:
        s = os.path.join(CSRC, src)
        o = os.path.join(obj_dir, src.replace(".cu", ".o"))
        objs.append(o)
        if force or _stale(o, [s] + headers):
            nvcc = nvcc or _nvcc()
            cmd = [nvcc] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", s, "-o", o]
            procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = None
    for src, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0 and failed is None:
            failed = f"nvcc failed on {src}:\n{out}"
        if verbose:
            print(out)
    if failed:
        raise RuntimeError(failed)
    if force or procs or _stale(target, objs):
        part = target + ".part"                            # never leave a half-written library behind
        cmd = [nvcc or _nvcc(), "-shared", "-o", part] + objs + ["-gencode", "arch=compute_100a,code=sm_100a"]
        r = subprocess.run(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}")
        os.replace(part, target)
    return target


if __name__ == "__main__":
    for name in [a for a in sys.argv[1:] if a in LIBRARIES] or list(LIBRARIES):
        print(build_library(force="--force" in sys.argv, verbose="--verbose" in sys.argv, which=name))
