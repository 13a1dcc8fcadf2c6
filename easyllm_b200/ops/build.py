"""In-tree build of the sm_100a kernel library (``libeasyllm_b200.so``) with nvcc.

Every ``csrc/*.cu`` is compiled for ``compute_100a/sm_100a`` (cross-compiles without a GPU)
and linked into one shared object beside this file, which ``ops.cuda`` loads with ctypes.
The entry points are plain ``extern "C"`` launchers taking raw device pointers and a CUDA
stream, so the library has no dependency on the PyTorch C++ ABI and builds in seconds.

    python -m easyllm_b200.ops.build [--force] [--verbose]
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ_DIR = os.path.join(HERE, "_build")
LIB_PATH = os.path.join(HERE, "libeasyllm_b200.so")
# the kernels that serving a model loads and launches; `ensure_serving` builds these alone
SERVE_LIB_PATH = os.path.join(HERE, "libeasyllm_b200_serve.so")
SERVE_SOURCES = ("attn_rows", "elementwise", "flash_attn", "gemm", "gemm_pair", "infer_elementwise", "matvec", "norm",
                 "optim", "recurrent")
# sources whose fp32 results must keep full accuracy (no approximate exp / tanh / division)
ACCURATE_SOURCES = ("attn_rows", "infer_elementwise", "matvec", "recurrent")

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "--use_fast_math", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden"]


def _nvcc():
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found; set NVCC or put it on PATH")


def sources():
    return sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cu"))


def _digest(path, flags):
    h = hashlib.sha1(" ".join(flags).encode())
    for p in [path] + sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))):
        with open(p, "rb") as f:
            h.update(f.read())
    return h.hexdigest()


def _flags_for(base, extra_flags=()):
    drop = {"--use_fast_math"} if base in ACCURATE_SOURCES else set()
    return [f for f in NVCC_FLAGS if f not in drop] + list(extra_flags)


def _stale(only=None):
    """Sources (of the ``only`` base names, or all) whose object is missing or older than its sources and flags."""
    out = []
    for src in sources():
        base = os.path.splitext(os.path.basename(src))[0]
        if only is not None and base not in only:
            continue
        stamp = os.path.join(OBJ_DIR, base + ".o.sha1")
        if not os.path.exists(stamp) or open(stamp).read() != _digest(src, _flags_for(base)):
            out.append(base)
    return out


def ensure_serving():
    """Make sure a library with the serving kernels exists: the full one is brought up to date when it is there,
    otherwise the serving sources alone are compiled.  Returns the path ``ops.cuda`` will load."""
    if os.path.exists(LIB_PATH):
        return build() if os.path.isdir(OBJ_DIR) and _stale() else LIB_PATH
    return build(only=SERVE_SOURCES)


def build(force=False, verbose=False, extra_flags=(), only=None):
    """Compile stale objects in parallel and relink.  Returns the library path.  ``only``: base names of the sources of
    the serving library, which is then built instead of the full one."""
    os.makedirs(OBJ_DIR, exist_ok=True)
    nvcc = _nvcc()
    jobs, objs = [], []
    lib_path = LIB_PATH if only is None else SERVE_LIB_PATH
    for src in sources():
        base = os.path.splitext(os.path.basename(src))[0]
        if only is not None and base not in only:
            continue
        flags = _flags_for(base, extra_flags)
        obj = os.path.join(OBJ_DIR, base + ".o")
        stamp = obj + ".sha1"
        dig = _digest(src, flags)
        objs.append(obj)
        fresh = os.path.exists(obj) and os.path.exists(stamp) and open(stamp).read() == dig
        if force or not fresh:
            jobs.append((src, obj, stamp, dig, flags))

    def compile_one(job):
        src, obj, stamp, dig, flags = job
        cmd = [nvcc] + flags + (["-Xptxas", "-v"] if verbose else []) + ["-I", CSRC, "-c", src, "-o", obj]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode:
            raise RuntimeError(f"nvcc failed for {src}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            print(r.stderr)
        with open(stamp, "w") as f:
            f.write(dig)
        return src

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            for done in ex.map(compile_one, jobs):
                if verbose:
                    print("compiled", done)
    if jobs or not os.path.exists(lib_path) or any(os.path.getmtime(o) > os.path.getmtime(lib_path) for o in objs):
        part = f"{lib_path}.{os.getpid()}.tmp"          # another process may have the old library mapped
        cmd = [nvcc, "-shared", "-cudart", "static", "-o", part] + objs
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
        os.replace(part, lib_path)
    return lib_path


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
