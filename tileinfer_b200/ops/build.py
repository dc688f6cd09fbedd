"""Ahead-of-time build of the sm_100a kernels into in-tree shared libraries.

`nvcc` compiles the `csrc/*.cu` for compute_100a/sm_100a only and links one `libtileinfer_b200*.so` per group of
sources next to this file; a stamp with the hash of the sources and flags makes rebuilds a no-op.  There is
no JIT cache: the library is loaded with ctypes and its `extern "C"` launchers take raw device
pointers and a stream, so they can be captured into CUDA graphs.
"""
from __future__ import annotations

import concurrent.futures
import hashlib
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
BUILD = os.path.join(HERE, "build")

# One shared library per group of sources, so that a model is served after compiling only what it needs: "base" (products,
# sampling, pointwise ops) is used by every model family, the others by the family that has the mechanism.
GROUPS = {
    "base": ("gemm_tcgen05.cu", "lm_head.cu", "pointwise.cu", "sampling.cu", "symm.cu"),
    "rows": ("row_ops.cu",),
    "attention": ("attn_paged.cu", "attn_prefill.cu", "attn_general.cu"),
    "hybrid": ("fused_ar.cu", "gdn.cu", "gdn_chunk.cu", "gemv_w8a16.cu"),
    "latent": ("latent_ops.cu", "latent_attn.cu", "latent_decode.cu", "latent_prefill.cu"),
    "gla": ("gla.cu", "gla_chunk.cu"),
    "conv": ("conv.cu",),
    "delta": ("delta.cu", "delta_chunk.cu"),
    "ssd": ("ssd.cu", "ssd_chunk.cu"),
    "moe": ("moe_route.cu", "gemm_grouped.cu"),
}


def lib_path(group: str = "base", debug: bool = False) -> str:
    tail = ("" if group == "base" else "_" + group) + ("_dbg" if debug else "")
    return os.path.join(HERE, f"libtileinfer_b200{tail}.so")


LIB = lib_path()

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr",
              "-DTI_GEMV_WARPS=" + os.environ.get("TI_GEMV_WARPS", "16"),
              "-DTI_GEMV_TPS=" + os.environ.get("TI_GEMV_TPS", "8"),
              "-DTI_GEMM_RING_KB=" + os.environ.get("TI_GEMM_RING_KB", "192"),
              "-DTI_GEMV_PREFETCH_KB=" + os.environ.get("TI_GEMV_PREFETCH_KB", "0")]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    return "nvcc"


def sources(group: str = None) -> list:
    return [f for g, files in GROUPS.items() if group in (None, g) for f in files]


def _flags(debug: bool) -> list:
    return NVCC_FLAGS + (DEBUG_FLAGS if debug else [])


def _hash(group: str, debug: bool = False) -> str:
    """Hash of the flags, the group's sources and the headers."""
    h = hashlib.sha256(" ".join(_flags(debug)).encode())
    heads = [f for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    for f in sorted(heads + sources(group)):
        with open(os.path.join(CSRC, f), "rb") as fh:
            h.update(f.encode())
            h.update(fh.read())
    return h.hexdigest()


def _build_dir(debug: bool) -> str:
    return BUILD_DEBUG if debug else BUILD


def _stamp(group: str, debug: bool) -> str:
    return os.path.join(_build_dir(debug), f"stamp_{group}.txt")


def is_current(group: str = "base", debug: bool = False) -> bool:
    if not (os.path.exists(lib_path(group, debug)) and os.path.exists(_stamp(group, debug))):
        return False
    with open(_stamp(group, debug)) as f:
        return f.read().strip() == _hash(group, debug)


# The checked variant: every peer-buffer / KV-page / workspace index that comes from run-time data goes through
# TI_CHECK (common.cuh), which records kStatusBounds in the status word and SKIPS the access instead of faulting;
# TI_JITTER adds random __nanosleep delays before packet sends and collects (stress of the flag protocols).
# Selected at run time with TI_DEBUG_LIB=1 (see lib.py).
DEBUG_FLAGS = ["-DTI_BOUNDS_CHECK", "-DTI_JITTER"]
BUILD_DEBUG = os.path.join(HERE, "build_dbg")


def build(force: bool = False, verbose: bool = False, groups=None, debug: bool = False) -> str:
    """Compile (if needed) the given groups of sources (default: all) and return the path of the base library."""
    todo = [g for g in (groups or GROUPS) if force or not is_current(g, debug)]
    if not todo:
        return lib_path("base", debug)
    build_dir = _build_dir(debug)
    os.makedirs(build_dir, exist_ok=True)
    nvcc = _nvcc()
    extra = ["-Xptxas", "-v"] if verbose else []
    hashes = {g: _hash(g, debug) for g in todo}

    def one(src):
        obj = os.path.join(build_dir, src[:-3] + ".o")
        cmd = [nvcc, *_flags(debug), *extra, "-I", CSRC, "-c", os.path.join(CSRC, src), "-o", obj]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            sys.stderr.write(r.stderr)
        return obj

    with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 2)) as ex:
        jobs = {g: [ex.submit(one, s) for s in sources(g)] for g in todo}
        for g in todo:
            objs = [j.result() for j in jobs[g]]
            # linked under a temporary name and moved: a process that starts meanwhile never loads half a file
            tmp = f"{lib_path(g, debug)}.tmp{os.getpid()}"
            r = subprocess.run([nvcc, "-shared", "-o", tmp, *objs, "-lcudart"], capture_output=True, text=True)
            if r.returncode != 0:
                raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
            os.replace(tmp, lib_path(g, debug))
            with open(_stamp(g, debug), "w") as f:
                f.write(hashes[g])
    return lib_path("base", debug)


def build_debug(force: bool = False) -> str:
    """Compile the bounds-checked, jittered variant of every library (same sources, DEBUG_FLAGS)."""
    return build(force, debug=True)


if __name__ == "__main__":
    if "--debug" in sys.argv:
        print(build_debug(force="--force" in sys.argv))
    else:
        print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
