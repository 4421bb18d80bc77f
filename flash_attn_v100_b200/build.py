"""Build recipe for the sm_100a shared libraries (kept in-tree).

`libfa_b200.so` (csrc/*.cu) holds the attention operators and the operators of the Qwen3-style decoder; the hybrid
decoders share `libfa_b200_rows.so` (csrc/rows/*.cu, row-wise operators) and have their mixers in
`libfa_b200_hybrid.so` (csrc/hybrid/*.cu: decayed linear attention, latent attention) and `libfa_b200_mixers.so`
(csrc/mixers/*.cu: gated recurrences, chunked attention).  A process that serves one model builds and loads what that
model needs.

    python -m flash_attn_v100_b200.build            # rebuild what is out of date, all libraries
    python -m flash_attn_v100_b200.build --force
    python -m flash_attn_v100_b200.build -v         # also print ptxas resource usage

Every `.cu` file is compiled to an object of its own (in parallel, cached under
`_build/` by source time stamps and flags) and the objects of a library are linked
together.  nvcc cross-compiles without a GPU.  The libraries link only the CUDA
runtime (static); they have no libtorch dependency.
"""
from __future__ import annotations

import contextlib
import fcntl
import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

PKG_DIR = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG_DIR, "csrc")
INCLUDE = os.path.join(os.path.dirname(PKG_DIR), "include")
LIB_PATH = os.path.join(PKG_DIR, "libfa_b200.so")
OBJ_DIR = os.path.join(PKG_DIR, "_build")

COMPILE_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]
LINK_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-shared", "-Xcompiler", "-fPIC"]


LIBRARIES = {"attention": (LIB_PATH, CSRC)}
LIBRARIES.update({name: (os.path.join(PKG_DIR, f"libfa_b200_{name}.so"), os.path.join(CSRC, name))
                  for name in ("rows", "hybrid", "mixers")})


def sources(library: str = "attention"):
    folder = LIBRARIES[library][1]
    return sorted(os.path.join(folder, f) for f in os.listdir(folder) if f.endswith(".cu"))


def _headers():
    deps = [os.path.join(d, f) for _, d in LIBRARIES.values() for f in os.listdir(d) if f.endswith(".cuh")]
    deps += [os.path.join(INCLUDE, f) for f in os.listdir(INCLUDE)]
    return deps


def needs_build(lib_path: str = LIB_PATH, library: str = "attention") -> bool:
    if not os.path.exists(lib_path):
        return True
    t = os.path.getmtime(lib_path)
    return any(os.path.getmtime(d) > t for d in sources(library) + _headers())


@contextlib.contextmanager
def _build_lock():
    """One build at a time per checkout: processes that start together wait for the first one's result."""
    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(OBJ_DIR, "lock"), "w") as f:
        fcntl.flock(f, fcntl.LOCK_EX)
        yield


def find_nvcc() -> str:
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(nvcc):
        raise RuntimeError("nvcc not found: cannot build libfa_b200.so")
    return nvcc


def _run(cmd):
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError("nvcc failed:\n" + " ".join(cmd) + "\n" + res.stdout + res.stderr)
    return res.stderr


def build(force: bool = False, verbose: bool = False, extra_flags=None, lib_path: str = "",
          library: str = "attention") -> str:
    """Compile the sources of `library` that changed and link it (to `lib_path` if given).  `extra_flags` (or the
    environment variable FA_B200_NVCC_FLAGS) adds compiler flags, e.g. `-DFA_TC5_PROF` for the instrumented
    prefill kernel; objects built with different flags are cached side by side."""
    default_path = LIBRARIES[library][0]
    lib_path = lib_path or default_path
    extra = list(extra_flags) if extra_flags is not None else os.environ.get("FA_B200_NVCC_FLAGS", "").split()
    if not force and not extra and lib_path == default_path and not needs_build(lib_path, library):
        return lib_path
    nvcc = find_nvcc()
    with _build_lock():
        if not force and not extra and lib_path == default_path and not needs_build(lib_path, library):
            return lib_path          # another process built it meanwhile
        flags = COMPILE_FLAGS + extra + (["-Xptxas", "-v"] if verbose else [])
        tag = hashlib.sha1(" ".join(COMPILE_FLAGS + extra).encode()).hexdigest()[:10]
        hdr_time = max(os.path.getmtime(h) for h in _headers())
        jobs, objs = [], []
        for src in sources(library):
            obj = os.path.join(OBJ_DIR, f"{library}.{os.path.splitext(os.path.basename(src))[0]}.{tag}.o")
            objs.append(obj)
            stale = force or verbose or not os.path.exists(obj) or \
                os.path.getmtime(obj) < max(os.path.getmtime(src), hdr_time)
            if stale:
                jobs.append([nvcc, *flags, "-I", INCLUDE, "-c", src, "-o", obj])
        with ThreadPoolExecutor(max_workers=max(1, min(len(jobs), os.cpu_count() or 1))) as pool:
            logs = list(pool.map(_run, jobs))
        if verbose:
            sys.stderr.write("".join(logs))
        part = f"{lib_path}.{os.getpid()}.tmp"
        _run([nvcc, *LINK_FLAGS, "-o", part, *objs])
        os.replace(part, lib_path)   # a process that has the old file mapped keeps it
    return lib_path


if __name__ == "__main__":
    for name in LIBRARIES:
        print(build(force="--force" in sys.argv, verbose="-v" in sys.argv, library=name))
