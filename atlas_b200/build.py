"""Builds the native libraries in-tree with nvcc / g++ (no JIT cache):

* ``atlas_b200/_C/libatlas_b200_kernels.so``  — every ``csrc/*.cu`` compiled for sm_100a
* ``atlas_b200/_C/libatlas_b200_runtime.so``  — host runtime (``csrc/runtime/*.cpp``)
* ``atlas_b200/_C/libatlas_b200_bench.so``    — kernels that only the benchmarks use (``bench/csrc/*.cu``: memory-stream
  probes), kept out of the library the engine loads

``python -m atlas_b200.build`` rebuilds what is out of date.  nvcc cross-compiles without a GPU.
"""
from __future__ import annotations

import concurrent.futures as cf
import fcntl
import os
import shutil
import subprocess
import sys
from typing import List, Optional

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "_C")
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr"]
KERNEL_LIB = os.path.join(OUT, "libatlas_b200_kernels.so")
RUNTIME_LIB = os.path.join(OUT, "libatlas_b200_runtime.so")
BENCH_CSRC = os.path.join(HERE, "bench", "csrc")
BENCH_LIB = os.path.join(OUT, "libatlas_b200_bench.so")


def _nvcc() -> str:
    return shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"


def _newer(src: str, dst: str, extra: List[str]) -> bool:
    if not os.path.exists(dst):
        return True
    t = os.path.getmtime(dst)
    return any(os.path.getmtime(f) > t for f in [src] + extra)


def _run(cmd: List[str]) -> None:
    r = subprocess.run(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if r.returncode != 0:
        raise RuntimeError("command failed: " + " ".join(cmd) + "\n" + r.stdout)


# translation units every library holds, and those of the mixers, residual forms and activation types
_UNITS_BASE = ("runtime",)
_UNITS_BF16 = ("gemm", "elementwise", "attention", "attention_tc16")
_UNITS_F32 = ("attention_f32",)
_UNITS_LISTED = ("streams",)                   # residual forms of models that list their layers
_UNITS_OF_KIND = {"rglru": ("conv1d", "rglru"), "wkv": ("recurrent",), "parallel": ("recurrent", "conv1d"), "mamba2": ("recurrent", "conv1d"),
                  "mlstm": ("mlstm",), "latent_attention": ("latent",), "differential": ("differential",)}


def units_for(cfg) -> Optional[List[str]]:
    """Translation units (``csrc/<unit>.cu``) that a model given by ``cfg`` calls outside of sampling, or None for all of
    them.  Known for models that list their layers."""
    if not cfg.layer_specs or cfg.quant.method != "none":
        return None
    units = set(_UNITS_BASE + (_UNITS_F32 if cfg.dtype == "float32" else _UNITS_BF16) + _UNITS_LISTED)
    for i, spec in enumerate(cfg.layer_specs):
        units.update(_UNITS_OF_KIND.get(spec.kind, ()))
        if cfg.for_layer(i).qk_norm_rows:
            units.add("row_norm_kv")
        if cfg.is_moe_layer(i):
            units.add("moe")
    if cfg.input_conv_taps:
        units.add("conv1d")
    return sorted(units)


def _sources() -> List[str]:
    return sorted(f[:-3] for f in os.listdir(CSRC) if f.endswith(".cu"))


def _headers() -> List[str]:
    return [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]


def kernels_current() -> bool:
    """The full kernel library exists and is newer than its sources."""
    headers = _headers()
    return not any(_newer(os.path.join(CSRC, u + ".cu"), KERNEL_LIB, headers) for u in _sources())


def build_kernels(verbose: bool = False, ptxas_v: bool = False, units: Optional[List[str]] = None) -> str:
    """Compile what is out of date and link it: the full library, or one of the given translation units only."""
    os.makedirs(OUT, exist_ok=True)
    lib = KERNEL_LIB if units is None else os.path.join(OUT, "libatlas_b200_kernels_" + "_".join(units) + ".so")
    with open(os.path.join(OUT, ".lock"), "w") as lock:          # two processes of a fresh checkout build one after the other
        fcntl.flock(lock, fcntl.LOCK_EX)
        headers = _headers()
        objs, jobs = [], []
        for u in (_sources() if units is None else units):
            src, obj = os.path.join(CSRC, u + ".cu"), os.path.join(OUT, u + ".o")
            objs.append(obj)
            if _newer(src, obj, headers):
                jobs.append([_nvcc()] + NVCC_FLAGS + (["-Xptxas", "-v"] if ptxas_v else []) + ["-I", CSRC, "-c", src, "-o", obj])
        if jobs:
            if verbose:
                print(f"[atlas_b200.build] compiling {len(jobs)} CUDA file(s) for sm_100a", file=sys.stderr)
            with cf.ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
                list(ex.map(_run, jobs))
        if jobs or any(_newer(o, lib, []) for o in objs):
            _run([_nvcc(), "-shared", "-o", lib + ".part"] + objs + ["-lcudart"])
            os.replace(lib + ".part", lib)
    return lib


def build_runtime(verbose: bool = False) -> str:
    os.makedirs(OUT, exist_ok=True)
    rdir = os.path.join(CSRC, "runtime")
    if not os.path.isdir(rdir):
        return ""
    srcs = sorted(os.path.join(rdir, f) for f in os.listdir(rdir) if f.endswith(".cpp"))
    hdrs = [os.path.join(rdir, f) for f in os.listdir(rdir) if f.endswith(".h")]
    if not srcs:
        return ""
    if any(_newer(s, RUNTIME_LIB, hdrs) for s in srcs):
        if verbose:
            print("[atlas_b200.build] compiling host runtime", file=sys.stderr)
        _run(["g++", "-O2", "-std=c++17", "-fPIC", "-shared", "-pthread", "-o", RUNTIME_LIB] + srcs)
    return RUNTIME_LIB


def build_bench(verbose: bool = False) -> str:
    """Benchmark-only kernels; they use the kernel library's tensor-map helper, so that library is linked in."""
    if not os.path.isdir(BENCH_CSRC):
        return ""
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    cus = sorted(f for f in os.listdir(BENCH_CSRC) if f.endswith(".cu"))
    objs, stale = [], False
    for f in cus:
        src, obj = os.path.join(BENCH_CSRC, f), os.path.join(OUT, "bench_" + f[:-3] + ".o")
        objs.append(obj)
        if _newer(src, obj, headers):
            if verbose:
                print(f"[atlas_b200.build] compiling bench/csrc/{f}", file=sys.stderr)
            _run([_nvcc()] + NVCC_FLAGS + ["-I", CSRC, "-c", src, "-o", obj])
            stale = True
    if objs and (stale or not os.path.exists(BENCH_LIB)):
        _run([_nvcc(), "-shared", "-o", BENCH_LIB] + objs + ["-L", OUT, "-latlas_b200_kernels", "-Xlinker", "-rpath=$ORIGIN",
                                                             "-lcudart"])
    return BENCH_LIB


def build_all(verbose: bool = True) -> None:
    build_kernels(verbose)
    build_runtime(verbose)
    build_bench(verbose)


if __name__ == "__main__":
    build_all(True)
    print(KERNEL_LIB)
