"""Build libgptb200.so (the C-ABI library with the sm_100a kernels) in-tree with nvcc.

Usage:  python -m gpt_b200.build [--verbose] [--force]

nvcc cross-compiles for sm_100a without a GPU.  Every source becomes an object of its own (compiled in parallel, kept in
gpt_b200/build/ and reused while nothing it depends on has changed); the shared objects land in gpt_b200/lib/ next to the
sources so that they are found without any install step:

  libgptb200.so           everything
  libgptb200_decoder.so   only what serving a decoder model needs (the products and the decoder models), for programs that
                          find nothing built: see decoder_library()
"""
from __future__ import annotations

import fcntl
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJDIR = os.path.join(HERE, "build")
LIBDIR = os.path.join(HERE, "lib")
LIB = os.path.join(LIBDIR, "libgptb200.so")
DECODER_LIB = os.path.join(LIBDIR, "libgptb200_decoder.so")

ARCH_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a"]
DECODER_SOURCES = ["capi.cu", "decoder_model.cu"]
SOURCES = ["capi.cu", "backend_capi.cu", "b200_backend.cu", "gpt_model.cu", "noalloc.cu", "decoder_model.cu", "loader.cpp"]


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found: libgptb200.so cannot be built")
    return exe


def _flags() -> list[str]:
    return ["-std=c++17", "-O3", *ARCH_FLAGS, "-lineinfo", "-Xcompiler", "-fPIC", "-I", os.path.join(HERE, "..", "include"), "-I", CSRC,
            "-I", os.path.join(CSRC, "iface")]


def _dependencies(source: str) -> list[str]:
    """The source and every header of this repository that it includes, directly or not."""
    roots = [CSRC, os.path.join(CSRC, "iface"), os.path.join(HERE, "..", "include")]
    seen, todo = set(), [os.path.join(CSRC, source)]
    while todo:
        f = todo.pop()
        if f in seen:
            continue
        seen.add(f)
        with open(f) as fh:
            for line in fh:
                if line.startswith("#include \""):
                    name = os.path.basename(line.split('"')[1])
                    todo += [os.path.join(r, name) for r in roots if os.path.exists(os.path.join(r, name))][:1]
    return sorted(seen)


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _run(cmd: list[str], what: str, verbose: bool) -> None:
    res = subprocess.run(cmd, capture_output=True, text=True)
    if verbose or res.returncode != 0:
        sys.stderr.write(res.stdout + res.stderr)
    if res.returncode != 0:
        raise RuntimeError("nvcc failed building " + what)


def _objects(sources: list[str], verbose: bool, force: bool) -> list[str]:

    def one(src: str) -> str:
        obj = os.path.join(OBJDIR, os.path.splitext(src)[0] + ".o")
        if force or _stale(obj, _dependencies(src) + [os.path.abspath(__file__)]):
            part = f"{obj}.{os.getpid()}.part"
            _run([_nvcc(), *(["-Xptxas", "-v"] if verbose else []), *_flags(), "-c", os.path.join(CSRC, src), "-o", part], src, verbose)
            os.replace(part, obj)
        return obj

    with ThreadPoolExecutor(max_workers=min(len(sources), os.cpu_count() or 1)) as pool:
        return list(pool.map(one, sources))


def _link(target: str, sources: list[str], verbose: bool, force: bool) -> str:
    os.makedirs(LIBDIR, exist_ok=True)
    os.makedirs(OBJDIR, exist_ok=True)
    with open(os.path.join(OBJDIR, "lock"), "w") as lock:     # two processes that find nothing built: one builds
        fcntl.flock(lock, fcntl.LOCK_EX)
        deps = sorted({d for s in sources for d in _dependencies(s)})
        if force or _stale(target, deps + [os.path.abspath(__file__)]):
            objs = _objects(sources, verbose, force)
            part = f"{target}.{os.getpid()}.part"
            _run([_nvcc(), *ARCH_FLAGS, "-Xcompiler", "-fPIC", "-shared", "-o", part, *objs], os.path.basename(target), verbose)
            os.replace(part, target)
    return target


def build(verbose: bool = False, force: bool = False, out: str | None = None, defines: list[str] | None = None) -> str:
    """`out` / `defines`: build a variant of the library somewhere else with extra -D flags (kernel experiments)."""
    if out:
        cmd = [_nvcc(), *_flags(), "-shared", *[f"-D{d}" for d in (defines or [])], "-o", out, *[os.path.join(CSRC, s) for s in SOURCES]]
        _run(cmd, out, verbose)
        return out
    return _link(LIB, SOURCES, verbose, force)


def decoder_library() -> str:
    """Path of a library with the decoder models: the complete one when it is there and current, else the small one, built on
    demand."""
    if os.path.exists(LIB) and not _stale(LIB, sorted({d for s in SOURCES for d in _dependencies(s)})):
        return LIB
    return _link(DECODER_LIB, DECODER_SOURCES, False, False)


if __name__ == "__main__":
    print(build(verbose="--verbose" in sys.argv, force="--force" in sys.argv))
