"""Builds libckb200.so in-tree: nvcc for the .cu kernels (sm_100a only), gcc for the C host code.

Usage:  python c-kernel-engine_b200/build.py [--verbose] [--force] [--part layer-stack]
The object files go to c-kernel-engine_b200/build/, the library next to this file.  A part is a library of its own with one model
family and what it needs: quicker to build where nothing else is used.
"""
from __future__ import annotations

import concurrent.futures as cf
import os
import subprocess
import sys

PKG = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(PKG, "csrc")
OBJ = os.path.join(PKG, "build")
LIB = os.path.join(PKG, "libckb200.so")
PARTS = {
    # model family -> (library, sources)
    "layer-stack": ("libckb200_layer_stack.so", [
        "runtime.c", "staging.cu", "json_mini.c", "safetensors.c", "model.c", "model_stack.c", "model_stack_weights.c", "model_stack_mixers.c",
        "layer_stack_config.c", "linear_gemv.cu", "linear_f32.cu", "linear_tc.cu", "mixer_rows.cu", "mixer_recurrence.cu", "mixer_step.cu", "attention_latent.cu",
        "attention_portion.cu", "attention_window.cu"]),
}
CUDA_HOME = os.environ.get("CUDA_HOME", "/usr/local/cuda")
NVCC = os.path.join(CUDA_HOME, "bin", "nvcc")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr", "-Xptxas", "-v",
]
NVCC_FLAGS += os.environ.get("CKB_NVCC_EXTRA", "").split()       # e.g. -DCKB_TC_TRACE or -DCKB_STEP_TRACE for the in-kernel timeline recorders
CC_FLAGS = ["-O2", "-fPIC", "-std=c11", "-Wall", "-Wextra", "-Wno-unused-parameter", "-fms-extensions", f"-I{CUDA_HOME}/include"]


def _newer(src: str, dst: str, deps: list[str]) -> bool:
    if not os.path.exists(dst):
        return True
    t = os.path.getmtime(dst)
    return any(os.path.getmtime(p) > t for p in [src, *deps])


def library_for(family: str) -> str:
    """Path of a library that runs models of this family: the whole one when it is built and current, else the family's part (built here
    if need be)."""
    sources = [os.path.join(base, f) for base in (CSRC, os.path.join(PKG, "..", "include")) for f in os.listdir(base) if os.path.isfile(os.path.join(base, f))]
    if os.path.exists(LIB) and not any(os.path.getmtime(p) > os.path.getmtime(LIB) for p in sources):
        return LIB
    return build(part=family)


def build(verbose: bool = False, force: bool = False, part: str | None = None) -> str:
    os.makedirs(OBJ, exist_ok=True)
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    headers += [os.path.join(PKG, "..", "include", f) for f in os.listdir(os.path.join(PKG, "..", "include"))]
    headers.append(os.path.abspath(__file__))
    jobs = []
    objs = []
    lib, sources = PARTS[part] if part else (LIB, sorted(os.listdir(CSRC)))
    lib = os.path.join(PKG, lib)
    for f in sources:
        src = os.path.join(CSRC, f)
        if f.endswith(".cu"):
            obj = os.path.join(OBJ, f[:-3] + ".o")
            cmd = [NVCC, *NVCC_FLAGS, "-c", src, "-o", obj]
        elif f.endswith(".c"):
            obj = os.path.join(OBJ, f[:-2] + ".o")
            cmd = ["gcc", *CC_FLAGS, "-c", src, "-o", obj]
        else:
            continue
        objs.append(obj)
        if force or _newer(src, obj, headers):
            jobs.append((f, cmd))

    def run(job):
        name, cmd = job
        r = subprocess.run(cmd, capture_output=True, text=True)
        return name, r

    with cf.ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        for name, r in ex.map(run, jobs):
            if r.returncode != 0:
                sys.stderr.write(r.stdout + r.stderr)
                raise RuntimeError(f"compile failed: {name}")
            if verbose:
                sys.stderr.write(f"--- {name}\n{r.stderr}")
            with open(os.path.join(OBJ, name + ".ptxas.txt"), "w") as fh:
                fh.write(r.stderr)
    if jobs or not os.path.exists(lib) or any(os.path.getmtime(o) > os.path.getmtime(lib) for o in objs):
        link = [NVCC, "-shared", "-o", lib, *objs, "-cudart", "static", "-lpthread", "-ldl", "-lrt"]
        r = subprocess.run(link, capture_output=True, text=True)
        if r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
    if part:
        return lib
    # the two thin model-ABI libraries (same symbol names, different signatures: they cannot share one library)
    for name, src in (("libckb200_model_v7.so", "model_v7.c"), ("libckb200_model_api.so", "model_handle.c")):
        out = os.path.join(PKG, name)
        srcp = os.path.join(CSRC, "abi", src)
        if force or _newer(srcp, out, headers + [LIB]):
            cmd = ["gcc", *CC_FLAGS, "-shared", "-fvisibility=hidden", srcp, "-o", out, f"-L{PKG}", "-lckb200", "-Wl,-rpath,$ORIGIN"]
            r = subprocess.run(cmd, capture_output=True, text=True)
            if r.returncode != 0:
                sys.stderr.write(r.stdout + r.stderr)
                raise RuntimeError(f"compile failed: {src}")
    return LIB


if __name__ == "__main__":
    print(build(verbose="--verbose" in sys.argv, force="--force" in sys.argv, part=sys.argv[sys.argv.index("--part") + 1] if "--part" in sys.argv else None))
