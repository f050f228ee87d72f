"""Compiles csrc/*.cu into libkanso_cuda.so (sm_100a only) beside this file.

    python kanso-infer_b200/build.py [--force] [--verbose] [--model DIR]

nvcc cross-compiles without a GPU. Objects go to build/ (git-ignored); the shared
library stays in-tree so that it travels with the source tree to the GPU machine.

With --model only what the model in DIR needs is compiled, into libkanso_cuda_<class>.so: a host
that serves one model class need not wait for the others' kernels.
"""
from __future__ import annotations

import json
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB = os.path.join(HERE, "libkanso_cuda.so")

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr"]

# What a library that serves one model class is made of; the full library has every source.
CORE = ["ctx", "kv_pool", "glue", "model_api", "safetensors", "engine"]
DENSE = ["dense_model", "dense_rows", "gemv_dense", "gemm_dense"]  # the unquantised classes
MODEL_CLASSES = {
    "Revitar": ["revitar", *DENSE, "sigmoid_attention", "sigmoid_prefill"],
    "Migurax": ["migurax", *DENSE, "latent_attention", "softmax_prefill", "mlstm"],
}


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found: the cuda backend cannot be built")
    return exe


def _deps_mtime() -> float:
    hdrs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    hdrs.append(os.path.join(HERE, "..", "include", "kanso_cuda.h"))
    return max(os.path.getmtime(h) for h in hdrs)


def model_class(model_dir: str) -> str:
    """The architecture that dir/config.json names; it must be a class with a source list."""
    with open(os.path.join(model_dir, "config.json")) as f:
        name = json.load(f).get("architecture")
    if name not in MODEL_CLASSES:
        raise RuntimeError(f"unknown architecture {name!r} (known: {', '.join(MODEL_CLASSES)})")
    return name


def current(lib: str, srcs) -> bool:
    """The library exists and no source of it is newer."""
    return os.path.exists(lib) and os.path.getmtime(lib) >= max(
        _deps_mtime(), *(os.path.getmtime(os.path.join(CSRC, s)) for s in srcs))


def build_for_model(model_dir: str) -> str:
    """The library to serve the model in `model_dir` with: the full one when it is up to date,
    else one of the model's own class, compiled if need be."""
    name = model_class(model_dir)
    if current(LIB, [f for f in os.listdir(CSRC) if f.endswith(".cu")]):
        return LIB
    srcs = [s + ".cu" for s in CORE + MODEL_CLASSES[name]]
    lib = os.path.join(HERE, f"libkanso_cuda_{name.lower()}.so")
    return lib if current(lib, srcs) else build(srcs=srcs, lib=lib)


def build(force: bool = False, verbose: bool = False, srcs=None, lib: str = LIB) -> str:
    os.makedirs(OBJ, exist_ok=True)
    srcs = sorted(srcs or [f for f in os.listdir(CSRC) if f.endswith(".cu")])
    hdr_t = _deps_mtime()
    nvcc = _nvcc()
    jobs = []
    for s in srcs:
        src, obj = os.path.join(CSRC, s), os.path.join(OBJ, s[:-3] + ".o")
        if force or not os.path.exists(obj) or os.path.getmtime(obj) < max(os.path.getmtime(src),
                                                                           hdr_t):
            cmd = [nvcc, *NVCC_FLAGS, "-c", src, "-o", obj]
            if verbose:
                cmd[1:1] = ["-Xptxas", "-v"]
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0 or verbose:
            sys.stderr.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
        if r.returncode != 0:
            raise RuntimeError("nvcc failed on " + cmd[-3])

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            list(ex.map(run, jobs))
    objs = [os.path.join(OBJ, s[:-3] + ".o") for s in srcs]
    if jobs or force or not os.path.exists(lib) or \
            os.path.getmtime(lib) < max(os.path.getmtime(o) for o in objs):
        # -z defs: a symbol that no object defines fails the build here, not the first dlopen
        run([nvcc, "-shared", "-o", lib, *objs, "-gencode", "arch=compute_100a,code=sm_100a",
             "-Xlinker", "-z", "-Xlinker", "defs"])
    return lib


if __name__ == "__main__":
    if "--model" in sys.argv:
        print(build_for_model(sys.argv[sys.argv.index("--model") + 1]))
    else:
        print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
