"""Build libb200p.so in-tree with nvcc for sm_100a.

Every csrc/*.cu is compiled to an object next to the library (in parallel) and
linked into lib/libb200p.so.  Objects are rebuilt when the source or any header
under include/ or csrc/ is newer.

build_decoder(architecture) links only what one decoder of the runtime needs, as
lib/libb200p_<architecture>.so: the command-line programs use it in a checkout
where the whole library has not been built.
"""
from __future__ import annotations

import glob
import os
import subprocess
from concurrent.futures import ThreadPoolExecutor

PKG = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(PKG)
CSRC = os.path.join(PKG, "csrc")
LIBDIR = os.path.join(PKG, "lib")
LIB = os.path.join(LIBDIR, "libb200p.so")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--expt-relaxed-constexpr", "-Xcompiler", "-fPIC",
    "-I" + os.path.join(ROOT, "include"), "-I" + CSRC,
]


# the sources every decoder of the runtime needs, and each decoder's own
RUNTIME = ("core", "tensor_map", "gemm_tc", "model_loader", "runtime")
DECODERS = {"Llama": ("decoder_gqa", "decode", "prefill"), "Maposun": ("decoder_latent", "latent_attn", "latent_prefill"),
            "Vofusun": ("decoder_hybrid", "grouped_attn", "grouped_prefill", "delta_rule")}


def _newest_header() -> float:
    hs = glob.glob(os.path.join(ROOT, "include", "**", "*.*"), recursive=True)
    hs += glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.hpp"))
    return max(os.path.getmtime(h) for h in hs)


def build(force: bool = False, verbose: bool = False) -> str:
    return _build(sorted(glob.glob(os.path.join(CSRC, "*.cu"))), LIB, force, verbose)


def current(lib: str = LIB) -> bool:
    """Whether the library is there and no source or header is newer."""
    srcs = glob.glob(os.path.join(CSRC, "*.cu"))
    return os.path.exists(lib) and os.path.getmtime(lib) >= max([_newest_header()] + [os.path.getmtime(s) for s in srcs])


def build_decoder(architecture: str, verbose: bool = False) -> str:
    """The path of a library that runs this decoder: the whole one if it is up to date, else one with just its sources."""
    if current():
        return LIB
    names = RUNTIME + DECODERS[architecture]
    return _build([os.path.join(CSRC, n + ".cu") for n in names], os.path.join(LIBDIR, f"libb200p_{architecture.lower()}.so"), False, verbose)


def _build(srcs, lib: str, force: bool, verbose: bool) -> str:
    os.makedirs(LIBDIR, exist_ok=True)
    hdr = _newest_header()
    jobs, objs = [], []
    for s in srcs:
        o = os.path.join(LIBDIR, os.path.basename(s)[:-3] + ".o")
        objs.append(o)
        if force or not os.path.exists(o) or os.path.getmtime(o) < max(os.path.getmtime(s), hdr):
            jobs.append(["nvcc", *NVCC_FLAGS, "-c", s, "-o", o])
    if jobs:
        def run(cmd):
            if verbose:
                print(" ".join(cmd), flush=True)
            subprocess.run(cmd, check=True)
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            list(ex.map(run, jobs))
    if jobs or not os.path.exists(lib) or os.path.getmtime(lib) < max(os.path.getmtime(o) for o in objs):
        cmd = ["nvcc", "-shared", "-o", lib, *objs, "-lcublas", "-Xlinker", "-rpath=/usr/local/cuda/lib64"]
        if verbose:
            print(" ".join(cmd), flush=True)
        subprocess.run(cmd, check=True)
    return lib


if __name__ == "__main__":
    print(build(verbose=True))
