"""Builds libdc_b200.so in-tree with nvcc for sm_100a.

    python -m densecore_b200.build [--force] [--verbose]

The library is plain CUDA C++ behind a C ABI (include/dc_b200.h); it does not
link against PyTorch.
"""
from __future__ import annotations

import glob
import os
import subprocess
import sys

PKG = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG, "csrc")
ROOT = os.path.dirname(PKG)
LIB = os.path.join(PKG, "libdc_b200.so")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden",
    "--expt-relaxed-constexpr",
]


# Sources of the layer-list decoders alone (no K-quant kernels): what a process that serves only such a model compiles.
PARTS = {"layers": ["api", "ffn_moe", "kv", "linear", "linear_tc", "misc", "mix_gqa", "mix_latent", "mix_lightning", "mix_recur", "model", "norm_act", "stack", "stack_config",
                    "stack_load"]}


def sources() -> list[str]:
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")))


def _stale(lib: str = LIB) -> bool:
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = sources() + glob.glob(os.path.join(CSRC, "*.h")) + glob.glob(os.path.join(CSRC, "*.cuh"))
    deps += glob.glob(os.path.join(ROOT, "include", "*.h"))
    return any(os.path.getmtime(d) > t for d in deps)


def nvcc() -> str:
    for c in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if c and (os.path.isabs(c) and os.path.exists(c) or not os.path.isabs(c)):
            return c
    return "nvcc"


def build(force: bool = False, verbose: bool = False, out: str | None = None, extra: list[str] | None = None) -> str:
    """out / extra: build a variant (extra nvcc flags) to another path, e.g. for A/B timing."""
    if out or extra:
        return _build_variant(out or LIB, extra or [])
    if not force and not _stale():
        return LIB
    objs = []
    procs = []
    os.makedirs(os.path.join(PKG, "build"), exist_ok=True)
    for src in sources():
        obj = os.path.join(PKG, "build", os.path.basename(src)[:-3] + ".o")
        cmd = [nvcc(), *NVCC_FLAGS, "-I", os.path.join(ROOT, "include"), "-c", src, "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
        objs.append(obj)
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0 or verbose:
            sys.stderr.write(f"--- {os.path.basename(src)}\n{out}\n")
        failed |= p.returncode != 0
    if failed:
        raise RuntimeError("nvcc failed")
    link = [nvcc(), "-shared", "-o", LIB, *objs, "-gencode", "arch=compute_100a,code=sm_100a", "-lcuda", "-ldl"]
    subprocess.check_call(link)
    return LIB


def build_part(part: str) -> str:
    """The whole library if it is built and up to date, else a library of one part's sources."""
    if not _stale():
        return LIB
    out = os.path.join(PKG, f"libdc_b200_{part}.so")
    if _stale(out):
        tmp = f"{out}.{os.getpid()}"
        _build_variant(tmp, [], [os.path.join(CSRC, f"{n}.cu") for n in PARTS[part]])
        os.replace(tmp, out)     # a process that starts meanwhile sees the old file or the finished one
    return out


def _build_variant(out: str, extra: list[str], srcs: list[str] | None = None) -> str:
    import shutil
    import tempfile
    tmp = tempfile.mkdtemp(prefix="dcb200_")
    try:
        return _compile(out, extra, srcs or sources(), tmp)
    finally:
        shutil.rmtree(tmp, ignore_errors=True)


def _compile(out: str, extra: list[str], srcs: list[str], tmp: str) -> str:
    objs, procs = [], []
    for src in srcs:
        obj = os.path.join(tmp, os.path.basename(src)[:-3] + ".o")
        cmd = [nvcc(), *NVCC_FLAGS, *extra, "-I", os.path.join(ROOT, "include"), "-c", src, "-o", obj]
        procs.append(subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True))
        objs.append(obj)
    for p in procs:
        o, _ = p.communicate()
        if p.returncode != 0:
            raise RuntimeError(o)
    subprocess.check_call([nvcc(), "-shared", "-o", out, *objs, "-gencode", "arch=compute_100a,code=sm_100a", "-lcuda", "-ldl"])
    return out


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
