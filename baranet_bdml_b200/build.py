"""Builds the C-ABI library in-tree with nvcc for sm_100a: one object per source, compiled side by side, then linked.

    python -m baranet_bdml_b200.build [--force] [--verbose]

`build()` makes libbn_attn.so, all of it.  `build_for(architecture)` is for a checkout in which nothing has been built:
it compiles only the sources that one model family launches and links them into a library of their own
(libbn_attn_<family>.so); objects are shared, so a later full build compiles the rest."""
from __future__ import annotations

import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libbn_attn.so")
OBJ = os.path.join(HERE, "build")
SOURCES = ["api.cu", "tma.cu", "attn_f32.cu", "rmsnorm.cu", "embed_argmax.cu", "kv_cache.cu", "attn_decode.cu",
           "attn_prefill_sm100.cu", "gemm_bf16_sm100.cu", "gemm_skinny.cu", "exchange.cu", "residual_norm.cu",
           "attn_portion.cu", "attn_portion_sm100.cu", "latent_attn.cu", "latent_decode.cu", "mamba2.cu", "ssd_scan.cu", "mm_f32.cu",
           "hyper_norm.cu", "gqa_chunk.cu"]
# what a model family launches
FAMILIES = {
    "soluzen": ["api.cu", "tma.cu", "mm_f32.cu", "embed_argmax.cu", "gemm_bf16_sm100.cu", "gemm_skinny.cu", "residual_norm.cu",
                "attn_portion.cu", "attn_portion_sm100.cu", "latent_attn.cu", "latent_decode.cu", "mamba2.cu", "ssd_scan.cu"],
    "duponex": ["api.cu", "tma.cu", "mm_f32.cu", "embed_argmax.cu", "gemm_bf16_sm100.cu", "gemm_skinny.cu", "hyper_norm.cu",
                "attn_portion.cu", "attn_portion_sm100.cu", "gqa_chunk.cu"],
}
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "--expt-relaxed-constexpr", "-Xcompiler", "-fPIC,-fvisibility=hidden",
              "-I" + os.path.join(ROOT, "include"), "-I" + CSRC]


def _headers():
    return [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cuh")] + \
           [os.path.join(ROOT, "include", "bn_attn.h"), __file__]


def _newer(target: str, deps) -> bool:
    """Whether `target` exists and is at least as new as every dependency."""
    if not os.path.exists(target):
        return False
    t = os.path.getmtime(target)
    return all(os.path.getmtime(d) <= t for d in deps)


def _run(cmd, verbose: bool) -> None:
    env = dict(os.environ)
    # the image exports CC/CXX wrappers that lack some spec files; nvcc should use the system g++
    env.pop("CC", None)
    env.pop("CXX", None)
    res = subprocess.run(cmd, env=env, capture_output=True, text=True)
    if verbose or res.returncode != 0:
        sys.stderr.write(res.stdout + res.stderr)
    if res.returncode != 0:
        raise RuntimeError("nvcc failed: " + " ".join(cmd))


def _build(sources, out: str, force: bool, verbose: bool, extra_flags) -> str:
    paths = [os.path.join(CSRC, s) for s in sources]
    headers = _headers()
    if not force and not extra_flags and _newer(out, paths + headers):
        return out
    nvcc = os.environ.get("NVCC", "nvcc")
    # objects of a build with extra flags are not the ordinary ones
    obj_dir = OBJ if not extra_flags else out + ".obj"
    os.makedirs(obj_dir, exist_ok=True)

    def compile_one(src):
        obj = os.path.join(obj_dir, os.path.basename(src)[:-3] + ".o")
        if force or extra_flags or not _newer(obj, [src] + headers):
            part = f"{obj}.{os.getpid()}.part.o"            # a concurrent build never links half an object
            _run([nvcc] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + list(extra_flags) + ["-c", src, "-o", part],
                 verbose)
            os.replace(part, obj)
        return obj

    with ThreadPoolExecutor(max_workers=min(len(paths), os.cpu_count() or 1)) as pool:
        objs = list(pool.map(compile_one, paths))
    part = f"{out}.{os.getpid()}.part.so"
    _run([nvcc] + NVCC_FLAGS[:2] + ["-shared", "-Xcompiler", "-fPIC"] + objs + ["-o", part], verbose)
    os.replace(part, out)
    return out


def build(force: bool = False, verbose: bool = False, extra_flags=(), out: str = LIB) -> str:
    return _build(SOURCES, out, force, verbose, list(extra_flags))


def family_lib(family: str) -> str:
    return os.path.join(HERE, f"libbn_attn_{family}.so")


def build_for(family: str) -> str:
    """The library a model of `family` needs, compiled if it has to be: the full one where it is up to date, else the
    family's own."""
    if _newer(LIB, [os.path.join(CSRC, s) for s in SOURCES] + _headers()):
        return LIB
    if family not in FAMILIES:
        return build()
    return _build(FAMILIES[family], family_lib(family), False, False, [])


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
