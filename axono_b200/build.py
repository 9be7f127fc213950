"""Builds the C-ABI library (axono_b200/lib/libaxono_b200.so) for sm_100a with nvcc, and the native
Python module `libaxono` (host runtime + operator adapters + pybind11 binding) that links against it.

    python -m axono_b200.build [--force] [--verbose] [--serving DESIGN]

nvcc cross-compiles without a GPU; the library is kept in-tree so it travels with the
source checkout.  Sources compile to objects side by side and only where a source or header is newer.

`build_serving()` links the subset of the same objects that serving a language model calls into a library of its own
(libaxono_b200_lm_<design>.so): a fresh checkout that only serves a model compiles that much and no more.
"""
from __future__ import annotations

import concurrent.futures
import contextlib
import fcntl
import glob
import os
import shutil
import subprocess
import sys

PKG = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(PKG)
CSRC = os.path.join(PKG, "csrc")
LIB_DIR = os.path.join(PKG, "lib")
OBJ_DIR = os.path.join(LIB_DIR, "obj")
LIB = os.path.join(LIB_DIR, "libaxono_b200.so")
# what serving any language model takes; a model class names the rest as `kernel_sources`
SERVING_SOURCES = ("core.cu", "fused.cu", "kv_arena.cu", "latent_attn.cu", "latent_prefill.cu", "latent_umma.cu", "linear_lt.cpp",
                   "residual_norm.cu")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC",
]


def sources():
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")) + glob.glob(os.path.join(CSRC, "*.cpp")))


def serving_lib(architecture: str) -> str:
    return os.path.join(LIB_DIR, f"libaxono_b200_lm_{architecture.lower()}.so")


def _headers():
    return (glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h")) +
            glob.glob(os.path.join(ROOT, "include", "*.h")))


def _newer(deps, target) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


@contextlib.contextmanager
def _build_lock():
    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(OBJ_DIR, ".lock"), "w") as f:
        fcntl.flock(f, fcntl.LOCK_EX)
        yield


def _link(lib: str, srcs, force: bool, verbose: bool) -> str:
    if not force and not _newer(list(srcs) + _headers(), lib):
        return lib
    with _build_lock():
        nvcc = os.environ.get("NVCC") or shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
        headers = _headers()

        def compile_one(src):
            obj = os.path.join(OBJ_DIR, os.path.basename(src) + ".o")
            if force or _newer([src] + headers, obj):
                cmd = [nvcc, *NVCC_FLAGS, "-I", os.path.join(ROOT, "include"), "-I", CSRC]
                if verbose:
                    cmd += ["-Xptxas", "-v"]
                part = f"{obj}.{os.getpid()}"
                subprocess.check_call([*cmd, "-c", src, "-o", part])
                os.replace(part, obj)
            return obj

        with concurrent.futures.ThreadPoolExecutor(max(1, min(len(srcs), os.cpu_count() or 1))) as pool:
            objs = list(pool.map(compile_one, srcs))
        part = f"{lib}.{os.getpid()}"
        subprocess.check_call([nvcc, *NVCC_FLAGS, "-shared", "-o", part, *objs, "-ldl"])
        os.replace(part, lib)
    return lib


def build(force: bool = False, verbose: bool = False) -> str:
    return _link(LIB, sources(), force, verbose)


def build_serving(architecture: str, kernel_sources=(), force: bool = False, verbose: bool = False) -> str:
    """The library a process that serves one design loads: the full one when it is there and up to date, else the subset."""
    if not force and not _newer(sources() + _headers(), LIB):
        return LIB
    srcs = [os.path.join(CSRC, name) for name in (*SERVING_SOURCES, *kernel_sources)]
    return _link(serving_lib(architecture), srcs, force, verbose)


HOST = os.path.join(CSRC, "host")


def native_module_path() -> str:
    import sysconfig

    return os.path.join(LIB_DIR, "libaxono" + sysconfig.get_config_var("EXT_SUFFIX"))


def build_native(force: bool = False) -> str:
    """The `libaxono` extension module: csrc/host/*.cpp compiled with g++ against pybind11, the CUDA
    runtime and the C-ABI library beside it (rpath $ORIGIN)."""
    import sysconfig

    import pybind11

    lib = build(force=force)
    out = native_module_path()
    srcs = sorted(glob.glob(os.path.join(HOST, "*.cpp")))
    deps = srcs + glob.glob(os.path.join(HOST, "*.h")) + glob.glob(os.path.join(ROOT, "include", "*.h")) + [lib]
    if not force and os.path.exists(out) and all(os.path.getmtime(d) <= os.path.getmtime(out) for d in deps):
        return out
    cuda_home = os.environ.get("CUDA_HOME", "/usr/local/cuda")
    cmd = [os.environ.get("CXX", "g++"), "-std=c++17", "-O2", "-fPIC", "-shared", "-fvisibility=hidden",
           "-I", os.path.join(ROOT, "include"), "-I", HOST, "-I", pybind11.get_include(),
           "-I", sysconfig.get_paths()["include"], "-I", os.path.join(cuda_home, "include"),
           "-o", out, *srcs,
           "-L", LIB_DIR, "-laxono_b200", "-L", os.path.join(cuda_home, "lib64"), "-lcudart", "-ldl",
           "-Wl,-rpath,$ORIGIN", "-Wl,-rpath," + os.path.join(cuda_home, "lib64")]
    subprocess.check_call(cmd)
    return out


if __name__ == "__main__":
    if "--serving" in sys.argv:
        from axono_b200.models import model_class

        design = sys.argv[sys.argv.index("--serving") + 1]
        print(build_serving(design, model_class(design).kernel_sources, "--force" in sys.argv, "--verbose" in sys.argv))
        sys.exit(0)
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
    print(build_native(force="--force" in sys.argv))
