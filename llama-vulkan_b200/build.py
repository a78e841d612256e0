"""Builds the native libraries of this package in-tree with nvcc / g++.

    python llama-vulkan_b200/build.py [--force] [--locked] [program ...]

Outputs (next to this file): liblv_b200.so (sm_100a kernels + C ABI),
libllava_host.so (C++ host surface) and the command-line tools vulkan_llama and trace_run.
"""
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
CSRC = os.path.join(HERE, "csrc")
HOST = os.path.join(HERE, "host")
PROGRAMS = [("main.cpp", "vulkan_llama"), ("trace_run.cpp", "trace_run")]

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--use_fast_math=false", "-Xcompiler", "-fPIC", "-Xcompiler", "-Wall",
]


def _nvcc():
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(nvcc):
        raise RuntimeError("nvcc not found")
    return nvcc


def _newer(target, sources):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(s) > t for s in sources)


def _run(cmd):
    print("+", " ".join(cmd), flush=True)
    subprocess.check_call(cmd)


def _glob(d, exts):
    return sorted(os.path.join(d, f) for f in os.listdir(d) if f.endswith(exts))


def build_kernels(force=False, verbose_ptxas=False):
    """Compiles every .cu file to an object of its own (in parallel, only the stale ones) and links them."""
    from concurrent.futures import ThreadPoolExecutor
    cu = _glob(CSRC, (".cu",))
    headers = _glob(CSRC, (".cuh", ".h")) + [os.path.join(ROOT, "include", "lv_b200.h")]
    out = os.path.join(HERE, "liblv_b200.so")
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    flags = [f for f in NVCC_FLAGS if f != "--use_fast_math=false"]
    if verbose_ptxas:
        flags += ["-Xptxas", "-v"]
    objs, stale = [], []
    for src in cu:
        obj = os.path.join(objdir, os.path.basename(src)[:-3] + ".o")
        objs.append(obj)
        if force or verbose_ptxas or _newer(obj, [src] + headers):
            stale.append((src, obj))
    with ThreadPoolExecutor(max_workers=max(1, min(len(stale), os.cpu_count() or 1))) as pool:
        list(pool.map(lambda so: _run([_nvcc(), "-c", "-o", so[1]] + flags + [so[0]]), stale))
    if stale or not os.path.exists(out):
        _run([_nvcc(), "-shared", "-o", out, "-gencode", "arch=compute_100a,code=sm_100a"] + objs + ["-lcudart", "-ldl"])
    return out


def build_host(force=False, programs=None):
    if not os.path.isdir(HOST):
        return None
    cpp = [f for f in _glob(HOST, (".cpp",)) if os.path.basename(f) not in [p[0] for p in PROGRAMS]] + _glob(os.path.join(HOST, "server"), (".cpp",))
    if not cpp:
        return None
    deps = cpp + _glob(HOST, (".h",)) + _glob(os.path.join(HOST, "server"), (".h",)) + [os.path.join(ROOT, "include", "lv_b200.h"), os.path.join(ROOT, "include", "llava_host.h")]
    deps = [d for d in deps if os.path.exists(d)]
    out = os.path.join(HERE, "libllava_host.so")
    cxx = shutil.which("g++") or "g++"
    if force or _newer(out, deps):
        _run([cxx, "-std=c++20", "-O2", "-fPIC", "-shared", "-pthread", "-Wall", "-o", out] + cpp +
             ["-L" + HERE, "-llv_b200", "-Wl,-rpath,$ORIGIN", "-Wl,-Bsymbolic"])
    for source, program in PROGRAMS:
        if programs is not None and program not in programs:
            continue
        main = os.path.join(HOST, source)
        exe = os.path.join(HERE, program)
        if force or _newer(exe, [main, out]):
            _run([cxx, "-std=c++20", "-O2", "-pthread", "-o", exe, main, "-L" + HERE, "-lllava_host", "-llv_b200",
                  "-Wl,-rpath,$ORIGIN"])
    return out


def build_all(force=False, programs=None):
    """programs: the command-line tools to link (all of them when None)."""
    k = build_kernels(force)
    h = build_host(force, programs)
    return k, h


if __name__ == "__main__":
    if "--locked" in sys.argv:          # programs that build on demand: one builder at a time
        import fcntl
        os.makedirs(os.path.join(HERE, "build"), exist_ok=True)
        lock = open(os.path.join(HERE, "build", ".lock"), "w")
        fcntl.flock(lock, fcntl.LOCK_EX)
    wanted = [p for _, p in PROGRAMS if p in sys.argv[1:]]
    build_all(force="--force" in sys.argv, programs=wanted or None)
