"""Builds libonellm_b200.so in-tree with nvcc for sm_100a (cross-compiles without a GPU).

    python -m onellm_b200.build [-v] [-f]            # the whole library
    python -m onellm_b200.build --design Finuvik     # only what serving that design needs (build/libonellm_finuvik.so)
"""
from __future__ import annotations

import json
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
ROOT = os.path.dirname(HERE)
LIB = os.path.join(HERE, "libonellm_b200.so")
OBJ_DIR = os.path.join(HERE, "build")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden", "--expt-relaxed-constexpr",
    "-I" + os.path.join(ROOT, "include"), "-I" + CSRC,
]

# What a design opened with onellm_model_open is linked from: the engine, the projections, sampling, and its own files.
ENGINE_SOURCES = ["elementwise.cu", "engine.cu", "errors.cpp", "gemm_tc.cu", "model_files.cpp", "norm.cu", "sampling.cu",
                  "skinny_gemm.cu", "skinny_gemm_staged.cu", "skinny_gemm_tc.cu", "weight_placer.cu"]
DESIGN_SOURCES = {
    "Finuvik": ["biased_attn.cu", "biased_attn_tc.cu", "finuvik.cu", "gated_recurrence.cu"],
    "Fuposun": ["biased_attn_tc.cu", "fuposun.cu", "gated_recurrence.cu", "latent_attn.cu", "latent_attn_tc.cu", "route.cu"],
}


def sources():
    return sorted(f for f in os.listdir(CSRC) if f.endswith((".cu", ".cpp")))


def _stale(target, deps):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _headers():
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    headers.append(os.path.join(ROOT, "include", "onellm_b200.h"))
    return headers


def _make(names, lib, verbose, force):
    os.makedirs(OBJ_DIR, exist_ok=True)
    headers = _headers()
    objs, procs = [], []
    for src in names:
        path = os.path.join(CSRC, src)
        obj = os.path.join(OBJ_DIR, os.path.splitext(src)[0] + ".o")
        objs.append(obj)
        if force or _stale(obj, [path] + headers):
            cmd = ["nvcc"] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-x", "cu", "-c", path, "-o", obj]
            procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0 or verbose:
            sys.stderr.write(f"--- {src}\n{out}\n")
        failed |= p.returncode != 0
    if failed:
        raise RuntimeError("nvcc failed")
    if force or procs or _stale(lib, objs):
        subprocess.check_call(["nvcc", "-shared", "-Wno-deprecated-gpu-targets", "-o", lib] + objs + ["-lcudart", "-ldl", "-lcurand"])
    return lib


def build(verbose: bool = False, force: bool = False) -> str:
    return _make(sources(), LIB, verbose, force)


def library_for(folder: str) -> str:
    """A library that serves the model in `folder`: the whole one when it is built and current, else one with only the
    files that model's design needs, compiled now if it has to be."""
    if not _stale(LIB, [os.path.join(CSRC, f) for f in sources()] + _headers()):
        return LIB
    with open(os.path.join(folder, "config.json")) as f:
        name = json.load(f).get("architecture")
    return build_design(name)


def build_design(name: str, verbose: bool = False, force: bool = False) -> str:
    if name not in DESIGN_SOURCES:
        return build(verbose, force)
    lib = os.path.join(OBJ_DIR, f"libonellm_{name.lower()}.so")
    return _make(ENGINE_SOURCES + DESIGN_SOURCES[name], lib, verbose, force)


if __name__ == "__main__":
    if "--design" in sys.argv:
        print(build_design(sys.argv[sys.argv.index("--design") + 1], verbose="-v" in sys.argv, force="-f" in sys.argv))
    else:
        print(build(verbose="-v" in sys.argv, force="-f" in sys.argv))
