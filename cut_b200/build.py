"""Builds libcutb.so (the C ABI + sm_100a kernels) in-tree with nvcc.

nvcc cross-compiles for sm_100a without a GPU, so this runs anywhere the CUDA
toolkit is installed.  The library lands next to this file so that it travels
with the source tree.
"""
from __future__ import annotations

import os
import shutil
import subprocess

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libcutb.so")
# layer operators and the layer-list models over dense bf16 weights: what a model without quantized weights needs
LAYER_SOURCES = ["cabi_layers.cu", "common.cu", "layer_ops.cu", "mixer_ops.cu", "dense_matvec.cu", "dense_gemm.cu", "window_attention.cu",
                 "latent_attention.cu", "moe.cu", "expert_matvec.cu"]
QUANT_SOURCES = ["cabi.cu", "qgemv_blocks.cu", "qmatmul_generic.cu", "dequant.cu", "transpose_q4.cu",
                 "qgemm_tc.cu", "qgemm_skinny.cu", "repack.cu", "attention.cu", "attention_prefill.cu", "qgemv_planes.cu"]
SOURCES = QUANT_SOURCES + LAYER_SOURCES
LAYERS_LIB = os.path.join(HERE, "libcutb_layers.so")
HEADERS = ["common.cuh", "kernels.h", "tcgen05.cuh", "qgemm_tc_common.cuh", "dense_common.cuh", "norm_stage.cuh",
           "attn_common.cuh", "moe_common.cuh",
           os.path.join("..", "..", "include", "cutb.h")]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC,-fvisibility=hidden"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _build(lib: str, sources: list[str], force: bool, verbose: bool) -> str:
    """Compile the stale objects of `sources` side by side and link `lib`.  Objects and library appear under their names only
    when complete, so two builds of one tree do not read each other's halves."""
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    hdrs = [os.path.join(CSRC, h) for h in HEADERS]
    objs, procs = [], []
    for src in sources:
        s = os.path.join(CSRC, src)
        o = os.path.join(objdir, src.replace(".cu", ".o"))
        objs.append(o)
        if force or _stale(o, [s] + hdrs):
            tmp = f"{o}.{os.getpid()}"
            cmd = [_nvcc(), *NVCC_FLAGS, "-c", s, "-o", tmp] + (["-Xptxas", "-v"] if verbose else [])
            procs.append((src, o, tmp, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = []
    for src, o, tmp, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0:
            failed.append(f"nvcc failed on {src}:\n{out}")
            continue
        os.replace(tmp, o)
        if verbose:
            print(out)
    if failed:
        raise RuntimeError("\n".join(failed))
    if force or procs or _stale(lib, objs):
        tmp = f"{lib}.{os.getpid()}"
        cmd = [_nvcc(), "-shared", "-o", tmp, *objs, "-Xcompiler", "-fPIC"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}{r.stderr}")
        os.replace(tmp, lib)
    return lib


def build(force: bool = False, verbose: bool = False) -> str:
    """Compile every .cu into an object (only the stale ones) and link libcutb.so."""
    return _build(LIB, SOURCES, force, verbose)


def build_layers(force: bool = False, verbose: bool = False) -> str:
    """The library a model without quantized weights runs on: libcutb.so if it is there and current, else libcutb_layers.so
    from the same objects without the quantized-matmul kernels (a fraction of the compile time)."""
    every = [os.path.join(CSRC, f) for f in SOURCES + HEADERS]
    if not force and not _stale(LIB, every):
        return LIB
    return _build(LAYERS_LIB, LAYER_SOURCES, force, verbose)


HOST_LIB = os.path.join(HERE, "libcut_host.so")
HOST_SOURCES = ["cut_api.cpp", "b200_compute.cpp", "gguf_upload.cpp", "llama_runner.cpp", "host_cabi.cpp"]


def _cuda_home() -> str:
    return os.path.dirname(os.path.dirname(_nvcc()))


def build_host(force: bool = False) -> str:
    """Compile the C++ host API (csrc/host) into libcut_host.so on top of libcutb.so."""
    build(force=force)
    hdir = os.path.join(CSRC, "host")
    srcs = [os.path.join(hdir, f) for f in HOST_SOURCES]
    deps = srcs + [os.path.join(hdir, "cut_api.h"), os.path.join(hdir, "gguf_upload.h"),
                   os.path.join(CSRC, "..", "..", "include", "cutb.h"), LIB]
    if force or _stale(HOST_LIB, deps):
        cuda = _cuda_home()
        cmd = ["g++", "-O2", "-std=c++17", "-fPIC", "-shared", "-o", HOST_LIB, *srcs, f"-I{cuda}/include",
               f"-L{cuda}/lib64", f"-L{HERE}", "-lcutb", "-lcudart_static", "-ldl", "-lrt", "-lpthread",
               "-Wl,-rpath,$ORIGIN"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"host build failed:\n{r.stdout}{r.stderr}")
    return HOST_LIB


if __name__ == "__main__":
    import sys

    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
    print(build_host(force="--force" in sys.argv))
