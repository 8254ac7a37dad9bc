"""Builds the native libraries in-tree.

* ``gcore_b200/ops/_gk_kernels.so``   - every CUDA kernel, compiled for sm_100a only.
* ``gcore_b200/runtime/_gk_runtime.so`` - host-side C++ runtime (rollout scheduler, KV block manager, bucket
  planner, sequence balancing); needs only g++.

The libraries export a plain C ABI and are loaded with ``ctypes`` (see ``gcore_b200/ops/_lib.py``); nothing is
JIT-compiled at run time, so a box without a compiler can run a tree that was built elsewhere.

Usage: ``python -m gcore_b200.build_native [--force] [--verbose]``
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parent
OPS_SRC = ROOT / "ops" / "csrc"
RT_SRC = ROOT / "runtime" / "csrc"
BUILD = ROOT.parent / "build"
KERNEL_LIB = ROOT / "ops" / "_gk_kernels.so"
RUNTIME_LIB = ROOT / "runtime" / "_gk_runtime.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo", "--use_fast_math",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
    "--expt-relaxed-constexpr",
]
# sources of models that promise 32-bit arithmetic where they say so: compiled without the approximate math functions
EXACT_MATH = {"conv_norm", "depth_average", "diff_attention", "diff_prefill", "latent_attention", "matrix_memory",
              "matrix_memory_chunk", "moe_serve", "router", "sandwich_norm", "scored_attention", "scored_prefill", "stream_mix",
              "window_attention", "window_prefill"}
# sources one served architecture needs: ``ensure_kernels`` builds only these when the full library is not there
KERNEL_SETS = {
    "nafitar": ("comm", "elementwise", "gemm_skinny", "gemm_tcgen05", "gemm_wide", "matrix_memory", "matrix_memory_chunk",
                "sample_filtered", "sandwich_norm", "vocab", "window_attention", "window_prefill"),
    "kedesun": ("attention_fwd", "comm", "depth_average", "elementwise", "gemm_skinny", "gemm_tcgen05", "gemm_wide",
                "latent_attention", "matrix_memory", "matrix_memory_chunk", "mla_decode", "moe_serve", "router",
                "sample_filtered", "sandwich_norm", "vocab", "window_attention"),
    "lobutar": ("attention_fwd", "comm", "diff_attention", "diff_prefill", "elementwise", "gemm_skinny", "gemm_tcgen05",
                "gemm_wide", "latent_attention", "mla_decode", "moe_serve", "router", "sample_filtered", "sandwich_norm",
                "stream_mix", "vocab", "window_attention"),
    "rezulorn": ("comm", "conv_norm", "elementwise", "gemm_skinny", "gemm_tcgen05", "gemm_wide", "matrix_memory",
                 "matrix_memory_chunk", "moe_serve", "sample_filtered", "scored_attention", "scored_prefill", "vocab",
                 "window_attention"),
}
CXX_FLAGS = ["-O2", "-std=c++17", "-fPIC", "-fvisibility=hidden", "-Wall", "-pthread"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


def _digest(paths) -> str:
    h = hashlib.sha256()
    for p in sorted(paths):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    return h.hexdigest()


def _run(cmd, verbose):
    if verbose:
        print(" ".join(map(str, cmd)), flush=True)
    r = subprocess.run(list(map(str, cmd)), capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"command failed: {' '.join(map(str, cmd))}\n{r.stdout}\n{r.stderr}")
    if verbose and (r.stdout or r.stderr):
        print(r.stdout, r.stderr)
    return r


def _stamp(lib: Path) -> Path:
    return lib.with_suffix(".stamp")   # beside the library, so that a copied tree keeps both


def _fresh(lib: Path, digest: str) -> bool:
    st = _stamp(lib)
    return lib.exists() and st.exists() and st.read_text() == digest


def _headers():
    return sorted(list(OPS_SRC.glob("*.cuh")) + list(OPS_SRC.glob("*.h")))


def _set_sources(name):
    return [OPS_SRC / f"{stem}.cu" for stem in KERNEL_SETS[name] if (OPS_SRC / f"{stem}.cu").exists()]


def build_kernels(force=False, verbose=False, ptxas_info=False, only=None) -> Path:
    """The kernel library of all sources, or with ``only`` (a key of ``KERNEL_SETS``) the library of that set."""
    srcs = _set_sources(only) if only else sorted(OPS_SRC.glob("*.cu"))
    target = KERNEL_LIB.with_name(f"_gk_kernels_{only}.so") if only else KERNEL_LIB
    hdrs = _headers()
    dig = _digest(srcs + hdrs)
    if not force and _fresh(target, dig):
        return target
    BUILD.mkdir(exist_ok=True)
    nvcc = _nvcc()
    hdr_dig = _digest(hdrs)

    def compile_one(src: Path) -> Path:
        obj = BUILD / (src.stem + ".o")
        ostamp = BUILD / (src.stem + ".sha")
        flags = [f for f in NVCC_FLAGS if not (f == "--use_fast_math" and src.stem in EXACT_MATH)]
        d = hashlib.sha256(src.read_bytes() + hdr_dig.encode() + " ".join(flags).encode()).hexdigest()
        if not force and obj.exists() and ostamp.exists() and ostamp.read_text() == d:
            return obj
        if ptxas_info:
            flags += ["-Xptxas", "-v"]
        r = _run([nvcc, *flags, "-I", OPS_SRC, "-c", src, "-o", obj], verbose)
        if ptxas_info:
            (BUILD / (src.stem + ".ptxas.txt")).write_text(r.stderr)
        ostamp.write_text(d)
        return obj

    with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 2)) as ex:
        objs = list(ex.map(compile_one, srcs))
    _link([nvcc, "-shared"], objs, ["-lcudart"], target, dig, verbose)
    return target


def _link(cmd, inputs, libs, target: Path, digest: str, verbose):
    """Links beside the target and moves into place, so that an interrupted build leaves no half-written library."""
    part = target.with_name(f".{target.stem}.{os.getpid()}.part")
    _run([*cmd, "-o", part, *inputs, *libs], verbose)
    os.replace(part, target)
    _stamp(target).write_text(digest)


def build_runtime(force=False, verbose=False) -> Path:
    srcs = sorted(RT_SRC.glob("*.cpp"))
    hdrs = sorted(RT_SRC.glob("*.h"))
    dig = _digest(srcs + hdrs)
    if not force and _fresh(RUNTIME_LIB, dig):
        return RUNTIME_LIB
    BUILD.mkdir(exist_ok=True)
    cxx = os.environ.get("CXX", "g++")
    _link([cxx, *CXX_FLAGS, "-shared"], srcs, [], RUNTIME_LIB, dig, verbose)
    return RUNTIME_LIB


def ensure_kernels(name: str) -> Path:
    """Kernel library that serves architecture ``name``: the full one when it is up to date, else the library of the
    architecture's own set, built now if need be.  Also brings the host runtime up to date.  Safe to call from several
    processes of one checkout."""
    import fcntl
    BUILD.mkdir(exist_ok=True)
    with open(BUILD / ".lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        build_runtime()
        if _fresh(KERNEL_LIB, _digest(sorted(OPS_SRC.glob("*.cu")) + _headers())):
            return KERNEL_LIB
        return build_kernels(only=name)


def build_all(force=False, verbose=False, ptxas_info=False):
    return build_kernels(force, verbose, ptxas_info), build_runtime(force, verbose)


if __name__ == "__main__":
    args = set(sys.argv[1:])
    libs = build_all("--force" in args, "--verbose" in args, "--ptxas" in args)
    for lib in libs:
        print(f"built {lib} ({lib.stat().st_size/1e6:.2f} MB)")
