#!/usr/bin/env python3
"""Build libvoxtral_b200.so in-tree with nvcc for sm_100a.

    python voxtral-tts.c_b200/build.py [--force] [--verbose-ptxas]
    python voxtral-tts.c_b200/build.py --lm     # only libvb200_lm.so: the decoder language models

The shared library lands next to this file (lib/libvoxtral_b200.so). It is built
for sm_100a only (-gencode arch=compute_100a,code=sm_100a); nvcc cross-compiles
without a GPU.
"""
import concurrent.futures
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIBDIR = os.path.join(HERE, "lib")
LIB = os.path.join(LIBDIR, "libvoxtral_b200.so")
LM_LIB = os.path.join(LIBDIR, "libvb200_lm.so")
OBJDIR = os.path.join(LIBDIR, "obj")

# the decoder language models (vb_lm.cu and what it uses) and the speech path; vb_tc.cu and
# vb_upload.cu serve both
LM_SOURCES = ["vb_tc.cu", "vb_upload.cu", "vb_lm.cu", "vb_lm_kernels.cu", "vb_lm_attn.cu", "vb_lm_latent.cu",
              "vb_lm_moe.cu", "vb_lm_delta.cu",
              "vb_lm_config.cpp", "vb_json.cpp", "vb_safetensors.cpp"]
SOURCES = LM_SOURCES + ["vb_engine.cu", "vb_simple.cu", "vb_model.cu", "vb_prefill.cu", "vb_abi.cu", "vb_noalloc.cu",
                        "vb_acoustic_tc.cu", "vb_batch.cu", "vb_stream.cu", "vb_codec.cu", "vb_synth.cpp"]
NVCC = os.environ.get("NVCC", "nvcc")
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-Wall"]


def _headers():
    hs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    inc = os.path.join(os.path.dirname(HERE), "include")
    hs += [os.path.join(inc, f) for f in os.listdir(inc) if f.endswith(".h")]
    return hs


def _stale(target, deps):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _run(cmd):
    print("+", " ".join(cmd), flush=True)
    subprocess.check_call(cmd)


def _compile(sources, force, verbose_ptxas):
    """Object files of the sources, stale ones rebuilt side by side."""
    os.makedirs(OBJDIR, exist_ok=True)
    headers = _headers()
    objs, jobs = [], []
    for src in sources:
        s = os.path.join(CSRC, src)
        o = os.path.join(OBJDIR, src + ".o")
        objs.append(o)
        if not (force or _stale(o, [s] + headers)):
            continue
        # written under a temporary name: an interrupted compiler leaves no half-written object behind
        tmp = f"{o}.{os.getpid()}.tmp"
        if src.endswith(".cu"):
            cmd = [NVCC, *NVCC_FLAGS, *(["-Xptxas", "-v"] if verbose_ptxas else []), "-c", s, "-o", tmp]
        else:
            cmd = ["g++", "-O3", "-std=c++17", "-fPIC", "-fopenmp", "-ffp-contract=off", "-Wall", "-c", s, "-o", tmp]
        jobs.append((cmd, tmp, o))

    def one(job):
        cmd, tmp, o = job
        _run(cmd)
        os.replace(tmp, o)

    with concurrent.futures.ThreadPoolExecutor(max_workers=os.cpu_count() or 1) as pool:
        list(pool.map(one, jobs))
    return objs


def _link(cmd, target):
    # link under a temporary name and rename: a reader never sees a half-written library
    tmp = f"{target}.{os.getpid()}.tmp"
    _run([*cmd, "-o", tmp])
    os.replace(tmp, target)


def build_lm(force=False):
    """libvb200_lm.so alone: the decoder language models without the speech path."""
    objs = _compile(LM_SOURCES, force, False)
    if force or _stale(LM_LIB, objs):
        _link([NVCC, "-shared", *objs, "-lcudart"], LM_LIB)
    return LM_LIB


def build(force=False, verbose_ptxas=False):
    objs = _compile(SOURCES, force, verbose_ptxas)
    # the synthetic-tensor generator also as a small library of its own: code that must not map
    # the CUDA library (the CPU reference arm of the benchmark) loads only this one
    synth_lib = os.path.join(LIBDIR, "libvb_synth.so")
    synth_obj = os.path.join(OBJDIR, "vb_synth.cpp.o")
    if force or _stale(synth_lib, [synth_obj]):
        _link(["g++", "-shared", synth_obj, "-fopenmp"], synth_lib)
    if force or _stale(LIB, objs):
        _link([NVCC, "-shared", *objs, "-Xcompiler", "-fopenmp", "-lcudart", "-lgomp"], LIB)
    return LIB


if __name__ == "__main__":
    if "--lm" in sys.argv:
        print(build_lm(force="--force" in sys.argv))
    else:
        build(force="--force" in sys.argv, verbose_ptxas="--verbose-ptxas" in sys.argv)
        print(LIB)
