"""tenzo_b200 — B200 (sm_100a) CUDA implementation of Tenzo's quantized decode path.

The product is ``lib/libtenzo_runtime.so``: hand-written CUDA kernels, a resident decode engine
and the C ABI of ``include/tenzo.h`` (+ ``tenzo_ext.h``, ``tenzo_kernels.h``). This Python package
is a thin ctypes layer over that library for tests and benchmarks; it adds no arithmetic and has
no CPU path — loading fails loudly if the library was not built.
"""
from __future__ import annotations

import ctypes as C
import json
import os
from pathlib import Path

from . import abi

__all__ = ["load_library", "load_library_for", "library_path", "abi"]

_PKG = Path(__file__).resolve().parent
_lib = None


def library_path(family: str | None = None) -> Path:
    return _PKG / "lib" / (f"libtenzo_{family}.so" if family else "libtenzo_runtime.so")


def load_library(build_if_missing: bool = True, family: str | None = None):
    """dlopen libtenzo_runtime.so and declare every prototype. Raises if it cannot be loaded.

    `family`: when the library with every model family is not there yet, a library with this one alone will do (built
    if missing); whichever was loaded first stays."""
    global _lib
    if _lib is not None:
        return _lib
    path = library_path()
    if not path.exists():
        if not build_if_missing:
            raise RuntimeError(f"{path} is missing: run `python -m tenzo_b200.build` (there is no CPU fallback)")
        from .build import build, build_family
        path = build_family(family) if family else build()
    L = C.CDLL(str(path), mode=os.RTLD_GLOBAL)
    abi.declare_tenzo_abi(abi.present(L))
    abi.declare_ext_abi(abi.present(L))
    abi.declare_kernel_abi(abi.present(L))
    _lib = L
    return L


def load_library_for(model_dir):
    """The library that serves the model in a folder (its config.json names the architecture)."""
    from .build import ARCHITECTURES
    try:
        arch = json.loads((Path(model_dir) / "config.json").read_text()).get("architecture")
    except (OSError, ValueError, AttributeError):
        arch = None                                        # opening the folder reports what is wrong with it
    return load_library(family=ARCHITECTURES.get(arch))
