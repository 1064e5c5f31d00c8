"""Builds libtlcuda.so in-tree with nvcc for sm_100a (no JIT cache, no pip install).

The whole library serves every model.  A part of it (PARTS) holds what one family of models needs and
becomes a library of its own, for callers that compile on first use (``ensure``).

    python -m tensorlogic_b200.build            # incremental
    python -m tensorlogic_b200.build --force
"""
from __future__ import annotations

import fcntl
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

PKG = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(PKG)
CSRC = os.path.join(PKG, "csrc")
INCLUDE = os.path.join(ROOT, "include")
OBJDIR = os.path.join(PKG, "build")
LIB = os.path.join(PKG, "libtlcuda.so")

PARTS = {
    "decoder": ("tlc_context", "tlc_qtensor", "tlc_attention", "tlc_gguf", "tlc_safetensors", "tlc_decoder", "tlc_dense_gemv",
                "tlc_dense_gemm", "tlc_dense_ops", "tlc_window_attention", "tlc_latent_attention", "tlc_latent_prefill",
                "tlc_decoder_streams"),
}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden,-Wall",
    "--expt-relaxed-constexpr",
    "-I", INCLUDE, "-I", CSRC,
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "bin", "nvcc"),
                 shutil.which("nvcc")):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found; libtlcuda cannot be built")


def sources() -> list[str]:
    return sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cu", ".cpp")))


def _deps_mtime() -> float:
    hdrs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    hdrs += [os.path.join(INCLUDE, f) for f in os.listdir(INCLUDE)]
    hdrs.append(os.path.abspath(__file__))
    return max(os.path.getmtime(h) for h in hdrs)


def build(force: bool = False, verbose: bool = False, extra: list[str] | None = None, part: str | None = None) -> str:
    """Compiles what has changed and links; returns the library's path."""
    os.makedirs(OBJDIR, exist_ok=True)
    with open(os.path.join(OBJDIR, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)  # two processes of a fresh checkout may ask at once
        return _build(force, verbose, extra, part)


def _object(src: str) -> str:
    return os.path.join(OBJDIR, os.path.splitext(os.path.basename(src))[0] + ".o")


def current() -> bool:
    """Is the whole library there and newer than everything it is made of?"""
    if not os.path.exists(LIB):
        return False
    m = os.path.getmtime(LIB)
    return m >= _deps_mtime() and all(m >= os.path.getmtime(src) for src in sources())


def ensure(part: str | None = None) -> str:
    """The library that serves ``part``: the whole one if it is current, else the part, built now."""
    return LIB if current() else build(part=part)


def _build(force: bool, verbose: bool, extra: list[str] | None, part: str | None) -> str:
    nvcc = _nvcc()
    hdr_m = _deps_mtime()
    env = dict(os.environ)
    # The image exports CC/CXX pointing at a wrapper without OpenMP specs; nvcc only needs a host g++.
    ccbin = shutil.which("g++") or "g++"
    jobs = []
    objs = []
    lib = os.path.join(PKG, f"libtlcuda_{part}.so") if part else LIB
    for src in sources():
        if part and os.path.splitext(os.path.basename(src))[0] not in PARTS[part]:
            continue
        obj = _object(src)
        objs.append(obj)
        if force or not os.path.exists(obj) or os.path.getmtime(obj) < max(os.path.getmtime(src), hdr_m):
            cmd = [nvcc, "-ccbin", ccbin, *NVCC_FLAGS, *(extra or []), "-x", "cu", "-c", src, "-o", obj]
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True, env=env)
        if verbose or r.returncode != 0:
            sys.stderr.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed on {cmd[-3]}")
        return r

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            list(ex.map(run, jobs))
    if jobs or force or not os.path.exists(lib) or os.path.getmtime(lib) < max(os.path.getmtime(o) for o in objs):
        run([nvcc, "-ccbin", ccbin, "-shared", "-o", lib, *objs, "-cudart", "static", "-ldl"])
    return lib


if __name__ == "__main__":
    path = build(force="--force" in sys.argv, verbose="-v" in sys.argv,
                 extra=["-Xptxas", "-v"] if "--ptxas" in sys.argv else None)
    print(path)
