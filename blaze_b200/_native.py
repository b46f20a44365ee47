"""Build and load the native libraries (in-tree, sm_100a only).

``libblaze_kernels.so``  — every ``csrc/kernels/*.cu`` (C ABI ``blz_*`` over raw device pointers and a stream,
                           returning a ``cudaError_t`` code, like the reference's kernel library,
                           ``kernels/CMakeLists.txt:23``).
``libblaze_runtime.so``  — ``csrc/runtime/*.cpp`` host runtime (safetensors reader, weight repack, page
                           allocator, CPU oracles, log bridge).

The reference builds its kernels with CMake and binds them through a Rust FFI crate
(``crates/blaze-sys/build.rs``, ``crates/blaze-sys/src/lib.rs``); here the binding is ctypes over the same kind
of C ABI.
"""
from __future__ import annotations

import ctypes
import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from typing import Dict, List, Optional, Sequence, Tuple

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CSRC = os.path.join(ROOT, "csrc")
LIBDIR = os.path.join(os.path.dirname(os.path.abspath(__file__)), "_lib")
KERNELS_SO = os.path.join(LIBDIR, "libblaze_kernels.so")
RUNTIME_SO = os.path.join(LIBDIR, "libblaze_runtime.so")
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC",
              "--expt-relaxed-constexpr", "-I" + os.path.join(CSRC, "include")]


def _nvcc() -> Optional[str]:
    for c in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if c and os.path.exists(c):
            return c
    return None


def _sources(sub: str, ext: str) -> List[str]:
    d = os.path.join(CSRC, sub)
    return sorted(os.path.join(d, f) for f in os.listdir(d) if f.endswith(ext)) if os.path.isdir(d) else []


def _digest(paths: List[str]) -> str:
    h = hashlib.sha256()
    incs = []
    for dp, _, fs in os.walk(os.path.join(CSRC, "include")):
        incs += [os.path.join(dp, f) for f in fs]
    for p in sorted(paths + incs):
        h.update(os.path.relpath(p, ROOT).encode())      # a library stays valid when the tree moves
        with open(p, "rb") as f:
            h.update(f.read())
    return h.hexdigest()


def _stale(so: str, paths: List[str]) -> bool:
    stamp = so + ".sha"
    if not os.path.exists(so) or not os.path.exists(stamp):
        return True
    with open(stamp) as f:
        return f.read().strip() != _digest(paths)


def _compile(cu: List[str], verbose: bool = False, force: bool = False) -> List[str]:
    """Object files of kernel sources; those whose source and headers have not changed are kept."""
    nvcc = _nvcc()
    if nvcc is None:
        raise RuntimeError("nvcc not found; cannot build blaze_b200 kernels")
    objdir = os.path.join(LIBDIR, "obj")
    os.makedirs(objdir, exist_ok=True)

    def one(src):
        obj = os.path.join(objdir, os.path.basename(src) + ".o")
        if not force and not _stale(obj, [src]):
            return obj
        cmd = [nvcc] + NVCC_FLAGS + ["-c", src, "-o", obj]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src}:\n{r.stdout}\n{r.stderr}")
        if verbose and r.stderr:
            print(r.stderr, file=sys.stderr)
        with open(obj + ".sha", "w") as f:
            f.write(_digest([src]))
        return obj

    # the longest compilations first, so that none of them starts when the others are done
    order = sorted(cu, key=lambda p: -os.path.getsize(p))
    with ThreadPoolExecutor(max_workers=min(max(os.cpu_count() or 8, 8), len(cu))) as ex:
        objs = list(ex.map(one, order))
    return sorted(objs)


def _link(so: str, cu: List[str], objs: List[str]) -> None:
    part = f"{so}.{os.getpid()}.part"
    r = subprocess.run([_nvcc(), "-shared", "-o", part] + objs + ["-gencode", "arch=compute_100a,code=sm_100a"],
                       capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    os.replace(part, so)
    with open(so + ".sha", "w") as f:
        f.write(_digest(cu))


def build_runtime(force: bool = False) -> None:
    """The host runtime library, if out of date."""
    os.makedirs(LIBDIR, exist_ok=True)
    cpp = _sources("runtime", ".cpp")
    if cpp and (force or _stale(RUNTIME_SO, cpp)):
        cxx = shutil.which("g++") or "g++"
        part = f"{RUNTIME_SO}.{os.getpid()}.part"
        cmd = [cxx, "-O3", "-std=c++17", "-fPIC", "-shared", "-pthread", "-mavx2", "-mfma", "-ffp-contract=off",
               "-I" + os.path.join(CSRC, "include"), "-o", part] + cpp
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"g++ failed:\n{r.stdout}\n{r.stderr}")
        os.replace(part, RUNTIME_SO)
        with open(RUNTIME_SO + ".sha", "w") as f:
            f.write(_digest(cpp))


def build(force: bool = False, verbose: bool = False) -> None:
    """Compile everything that is out of date.  Raises on a compiler error."""
    os.makedirs(LIBDIR, exist_ok=True)
    cu = _sources("kernels", ".cu")
    if cu and (force or _stale(KERNELS_SO, cu)):
        _link(KERNELS_SO, cu, _compile(cu, verbose, force))
    build_runtime(force)


def _part_so(sources: Sequence[str]) -> str:
    """A library of some of the kernel sources (names without ``.cu``), built if needed: what one model family launches, for a
    fresh checkout that has no complete library yet."""
    cu = [os.path.join(CSRC, "kernels", n + ".cu") for n in sorted(sources)]
    so = os.path.join(LIBDIR, "libblaze_kernels_" + hashlib.sha256(" ".join(sorted(sources)).encode()).hexdigest()[:8] + ".so")
    os.makedirs(LIBDIR, exist_ok=True)
    if _stale(so, cu):
        _link(so, cu, _compile(cu))
    return so


_kernels = None
_runtime = None


_parts: Dict[Tuple[str, ...], ctypes.CDLL] = {}


def kernels(sources: Optional[Sequence[str]] = None) -> ctypes.CDLL:
    """The CUDA kernel library.  Builds it when missing and nvcc is present; raises otherwise.  ``sources``: the kernel sources
    the caller launches from; while the complete library is missing or out of date, a library of just these is built."""
    global _kernels
    if sources is not None and _kernels is None and _stale(KERNELS_SO, _sources("kernels", ".cu")):
        key = tuple(sorted(sources))
        if key not in _parts:
            _parts[key] = ctypes.CDLL(_part_so(key))
        return _parts[key]
    if _kernels is None:
        if not os.path.exists(KERNELS_SO) or (os.environ.get("BLAZE_REBUILD") and _stale(KERNELS_SO, _sources("kernels", ".cu"))):
            build()
        if not os.path.exists(KERNELS_SO):
            raise RuntimeError(f"{KERNELS_SO} is missing: run `python -c 'import __graft_entry__ as g; g.build()'`")
        # BLAZE_KERNELS_SO: load another build of the kernel library (A/B timing of kernel variants in one process set-up)
        _kernels = ctypes.CDLL(os.environ.get("BLAZE_KERNELS_SO") or KERNELS_SO)
    return _kernels


def runtime() -> ctypes.CDLL:
    global _runtime
    if _runtime is None:
        if not os.path.exists(RUNTIME_SO):
            build_runtime()
        _runtime = ctypes.CDLL(RUNTIME_SO)
    return _runtime


def have_runtime() -> bool:
    try:
        runtime()
        return True
    except Exception:
        return False
