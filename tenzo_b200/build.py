"""Build libtenzo_runtime.so (the sm_100a CUDA kernels + engine + C ABI) in-tree with nvcc.

    python -m tenzo_b200.build            # build if stale
    python -m tenzo_b200.build --force

nvcc cross-compiles without a GPU. Flags that matter for results: -fmad=false (no silent FMA
contraction; the reference's CPU arithmetic rounds products and sums separately unless it uses an
explicit fused intrinsic) and no fast-math (IEEE division, sqrt, round-half-away).
"""
from __future__ import annotations

import argparse
import os
import subprocess
import sys
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
LIB = PKG / "lib" / "libtenzo_runtime.so"
# One library holds everything; a model family on its own can also be built as CORE + its sources (build_family).
CORE = ["engine_core.cu", "capi.cu", "sampler.cu", "model_registry.cu"]
FAMILIES = {
    "bitnet": ["tl1_gemv.cu", "tl1_umma.cu", "norm_quant.cu", "attention.cu", "attention_fast.cu", "lm_head.cu", "lm_head_umma.cu",
               "decode_persistent.cu", "engine.cu", "capi_bitnet.cu", "cuda_runtime_hal.cu", "model_loader.cu"],
    "hybrid": ["rows.cu", "gemm.cu", "gemm_umma.cu", "window_attention.cu", "window_attention_mma.cu", "linear_attention.cu", "linear_scan.cu",
               "delta_rule.cu", "latent_attention.cu", "route.cu", "hybrid_engine.cu", "hybrid_sozopel.cu", "hybrid_tigitar.cu"],
}
ARCHITECTURES = {"BitNet": "bitnet", "Sozopel": "hybrid", "Tigitar": "hybrid"}      # "architecture" of a model folder's config.json
SOURCES = CORE + FAMILIES["bitnet"] + FAMILIES["hybrid"]
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-fmad=false", "-Xcompiler", "-fPIC,-fvisibility=hidden,-O2", "-Xptxas", "-v",
]


def nvcc_path() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.sep not in cand or os.path.exists(cand)):
            return cand
    raise RuntimeError("nvcc not found")


def stale(lib: Path = LIB) -> bool:
    if not lib.exists():
        return True
    t = lib.stat().st_mtime
    deps = list(CSRC.glob("*.cu")) + list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h")) + \
        list((PKG.parent / "include").glob("*.h")) + [Path(__file__)]
    return any(d.stat().st_mtime > t for d in deps)


def build(force: bool = False, verbose: bool = False) -> Path:
    return _build(LIB, SOURCES, force, verbose)


def build_family(family: str, force: bool = False) -> Path:
    """The engine core with one model family: what a model of that family needs, and no more."""
    return _build(PKG / "lib" / f"libtenzo_{family}.so", CORE + FAMILIES[family], force, False)


def _build(lib: Path, sources: list[str], force: bool, verbose: bool) -> Path:
    if not force and not stale(lib):
        return lib
    objdir = lib.parent / ("obj" if lib == LIB else f"obj_{lib.stem}")
    objdir.mkdir(parents=True, exist_ok=True)
    nvcc = nvcc_path()
    procs = []
    for src in sources:
        obj = objdir / (src[:-3] + ".o")
        cmd = [nvcc, *NVCC_FLAGS, *os.environ.get("TENZO_NVCC_EXTRA", "").split(), "-c", str(CSRC / src), "-o", str(obj)]
        procs.append((src, obj, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    objs, log, failed = [], [], []
    for src, obj, p in procs:
        out, _ = p.communicate()
        log.append(f"== {src}\n{out}")
        if p.returncode != 0:
            failed.append(src)
        objs.append(str(obj))
    if failed:
        sys.stderr.write("\n".join(log))
        raise RuntimeError(f"nvcc failed on {', '.join(failed)}")
    (objdir.parent / ("ptxas.log" if lib == LIB else f"ptxas_{lib.stem}.log")).write_text("\n".join(log))
    if verbose:
        print("\n".join(log))
    part = lib.with_suffix(f".{os.getpid()}.part")             # a half-written library never carries the final name
    link = [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", str(part), *objs, "-cudart", "static"]
    r = subprocess.run(link, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if r.returncode != 0:
        sys.stderr.write(r.stdout)
        raise RuntimeError("link failed")
    os.replace(part, lib)
    return lib


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("-v", "--verbose", action="store_true")
    a = ap.parse_args()
    print(build(a.force, a.verbose))
