"""Builds the CUDA libraries with nvcc for sm_100a, in-tree, next to this file, so that they travel with the package:

    libperegrine_b200.so     the quantised path                        (include/peregrine_b200.h)
    libperegrine_b200_lm.so  the layers of the bf16 / f32 language models   (include/peregrine_b200_lm.h)

`python -m peregrine_b200.build` rebuilds both; `build("lm")` one of them; `ensure_built()` rebuilds only when a source
is newer than its library.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "lib", "obj")
LIB = os.path.join(HERE, "lib", "libperegrine_b200.so")
LIB_LM = os.path.join(HERE, "lib", "libperegrine_b200_lm.so")

CORE = ["pg_core.cu", "pg_sample.cu"]     # in both libraries

SOURCES = CORE + [
    "pg_api.cu",
    "pg_quantize.cu",
    "pg_gemm_naive.cu",
    "pg_gemv_w8a8.cu", "pg_gemv_wstream.cu",
    "pg_gemm_tcgen05.cu",
    "pg_gemm_tcgen05_2cta.cu",
    "pg_gguf.cu",
    "pg_gguf_stream.cu",
    "pg_noalloc.cu",
    "pg_w8a32.cu",
    "pg_peer.cu",
    "pg_llama.cu", "pg_llama_attn.cu",
    "pg_huffman.cu",
]

SOURCES_LM = CORE + [
    "pg_linear.cu", "pg_linear_gemv.cu", "pg_linear_tc.cu", "pg_linear_f32.cu",
    "pg_route.cu", "pg_rows.cu", "pg_delta.cu", "pg_scan.cu", "pg_attention.cu", "pg_attention_tc.cu", "pg_latent.cu",
]

# component -> (library, sources)
COMPONENTS = {"int8": (LIB, SOURCES), "lm": (LIB_LM, SOURCES_LM)}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden",
    # bit-exactness: IEEE division/sqrt, denormals kept; FMA contraction is avoided in the
    # kernels themselves through the *_rn intrinsics
    "--ftz=false", "--prec-div=true", "--prec-sqrt=true",
    "-I", os.path.join(ROOT, "include"), "-I", CSRC,
]


def _nvcc() -> str:
    for cand in (shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found; libperegrine_b200.so cannot be built")


def _deps():
    deps = [os.path.join(CSRC, f) for f in sorted(os.listdir(CSRC)) if f.endswith(".cuh")]
    return deps + [os.path.join(ROOT, "include", f) for f in ("peregrine_b200.h", "peregrine_b200_tune.h", "peregrine_b200_lm.h")] + [os.path.abspath(__file__)]


def is_stale(component: str = "int8") -> bool:
    lib, sources = COMPONENTS[component]
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    return any(os.path.getmtime(p) > t for p in [os.path.join(CSRC, s) for s in sources] + _deps())


def build(component: str = "", verbose: bool = False, ptxas_info: bool = False) -> str:
    """Compiles one component, or all of them; returns the (last) library's path."""
    nvcc = _nvcc()
    os.makedirs(OBJ, exist_ok=True)
    env = dict(os.environ)
    env.pop("CC", None)
    env.pop("CXX", None)
    wanted = [COMPONENTS[component]] if component else list(COMPONENTS.values())
    tag = f".{os.getpid()}"      # two builds at once do not write the same files

    def compile_one(src: str) -> str:
        obj = os.path.join(OBJ, src[:-3] + ".o")
        cmd = [nvcc, *NVCC_FLAGS, "-c", os.path.join(CSRC, src), "-o", obj + tag]
        if ptxas_info:
            cmd += ["-Xptxas", "-v"]
        r = subprocess.run(cmd, capture_output=True, text=True, env=env)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src}:\n{r.stdout}\n{r.stderr}")
        if verbose or ptxas_info:
            sys.stderr.write(r.stderr)
        os.replace(obj + tag, obj)
        return obj

    todo = list(dict.fromkeys(s for _, sources in wanted for s in sources))
    with ThreadPoolExecutor(max_workers=min(8, len(todo))) as ex:
        objs = dict(zip(todo, ex.map(compile_one, todo)))
    for lib, sources in wanted:
        cmd = [nvcc, "-shared", "-o", lib + tag, *[objs[s] for s in sources], "-gencode", "arch=compute_100a,code=sm_100a", "-Xcompiler", "-fPIC"]
        r = subprocess.run(cmd, capture_output=True, text=True, env=env)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
        os.replace(lib + tag, lib)
    return wanted[-1][0]


def ensure_built(component: str = "int8") -> str:
    if is_stale(component):
        build(component)
    return COMPONENTS[component][0]


if __name__ == "__main__":
    build(verbose=True, ptxas_info="--ptxas" in sys.argv)
    print("\n".join(lib for lib, _ in COMPONENTS.values()))
