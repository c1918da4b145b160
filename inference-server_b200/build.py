"""Builds libb200decode.so (the C-ABI library) in-tree with nvcc for sm_100a.

Run as a script (``python inference-server_b200/build.py``) or call
:func:`build_library`.  Only what is older than its source is compiled
again.  nvcc cross-compiles without a GPU present.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys

PKG_DIR = os.path.dirname(os.path.abspath(__file__))
ROOT_DIR = os.path.dirname(PKG_DIR)
CSRC = os.path.join(PKG_DIR, "csrc")
INCLUDE = os.path.join(ROOT_DIR, "include")
LIB_PATH = os.path.join(PKG_DIR, "libb200decode.so")
SOURCES = ["host.cu", "paged_attn.cu", "paged_prefill.cu", "paged_prefill_tc.cu", "decode_glue.cu", "dense_gemm.cu", "router_fused.cu", "moe_route.cu", "moe_gemm.cu",
           "moe_layer.cu", "ep_p2p.cu", "latent_attn.cu", "layer_glue.cu", "gated_glue.cu", "state_scan.cu", "mixed_attn.cu",
           "mixed_prefill_tc.cu", "state_step.cu", "state_chunk.cu"]
# Parts of the library that are enough for some model families, each with a library file of its own, for a process that
# has to build before it can run and needs no more than that.
SUBSETS = {
    "layered": ["host.cu", "paged_attn.cu", "paged_prefill.cu", "paged_prefill_tc.cu", "dense_gemm.cu", "latent_attn.cu",
                "layer_glue.cu"],
    "gated": ["host.cu", "dense_gemm.cu", "moe_route.cu", "layer_glue.cu", "gated_glue.cu", "state_scan.cu", "mixed_attn.cu",
              "mixed_prefill_tc.cu", "state_step.cu", "state_chunk.cu"],
}
HEADERS = ["common.cuh", "glue.cuh", "host.h"]
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-I", INCLUDE, "-I", CSRC,
]


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found; cannot build libb200decode.so")
    return exe


def _mtime(path: str) -> float:
    return os.path.getmtime(path) if os.path.exists(path) else 0.0


def _header_time() -> float:
    return max(_mtime(os.path.join(CSRC, h)) for h in HEADERS) if HEADERS else 0.0


def _newest(sources: list[str]) -> float:
    return max([_mtime(os.path.join(CSRC, f)) for f in sources]
               + [_header_time(), _mtime(os.path.join(INCLUDE, "b200_decode.h"))])


def _fresh(path: str, sources: list[str]) -> bool:
    return _mtime(path) >= _newest(sources)


def subset_path(subset: str) -> str:
    return LIB_PATH.replace(".so", f"_{subset}.so")


def build_library(force: bool = False, verbose: bool = False, subset: str | None = None) -> str:
    """Compile what is out of date of the .cu files under csrc/ (of one of SUBSETS if given) and link the shared library.
    Returns its path."""
    sources, lib_path = (SOURCES, LIB_PATH) if subset is None else (SUBSETS[subset], subset_path(subset))
    if not force and _fresh(lib_path, sources):
        return lib_path
    nvcc = _nvcc()
    obj_dir = os.path.join(ROOT_DIR, "build")
    os.makedirs(obj_dir, exist_ok=True)
    objs = []
    procs = []
    for src in sources:
        obj = os.path.join(obj_dir, src.replace(".cu", ".o"))
        objs.append(obj)
        if not force and _fresh(obj, [src]):
            continue
        cmd = [nvcc, *NVCC_FLAGS, "-c", os.path.join(CSRC, src), "-o", obj + ".tmp.o"]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        procs.append((src, obj, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    for src, obj, proc in procs:
        out, _ = proc.communicate()
        if verbose and out:
            print(out)
        if proc.returncode != 0:
            raise RuntimeError(f"nvcc failed on {src}:\n{out}")
        os.replace(obj + ".tmp.o", obj)
    tmp = lib_path + ".tmp"
    link = [nvcc, "-shared", "-o", tmp, *objs, "-gencode", "arch=compute_100a,code=sm_100a"]
    res = subprocess.run(link, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"link failed:\n{res.stdout}")
    os.replace(tmp, lib_path)
    return lib_path


def library_for(subset: str) -> str:
    """Path of an up-to-date library with the entry points of `subset`: the full one if it is there, else the subset's,
    built now if need be."""
    if _fresh(LIB_PATH, SOURCES):
        return LIB_PATH
    return build_library(subset=subset)


if __name__ == "__main__":
    path = build_library(force="--force" in sys.argv, verbose="-v" in sys.argv)
    print(path)
