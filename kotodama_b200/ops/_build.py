"""Builds and loads the native library (``csrc/*.cu`` -> ``kotodama_b200/_C/libkotodama_b200.so``).

The kernels are plain CUDA with ``extern "C"`` launchers (no PyTorch headers), compiled for
sm_100a only and called through ``ctypes`` with raw device pointers and the current stream.
"""
from __future__ import annotations

import ctypes
import os
import shutil
import subprocess
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path
from typing import Optional, Sequence

ROOT = Path(__file__).resolve().parents[2]
CSRC = ROOT / "csrc"
OUT_DIR = ROOT / "kotodama_b200" / "_C"
LIB = OUT_DIR / "libkotodama_b200.so"
OBJ_DIR = ROOT / "build" / "obj"

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden"]
# sources of the 32-bit mode (and of fp32 statistics) keep IEEE division, square roots and full-precision functions
PRECISE = {"block", "moe", "gemm_f32", "latent_attn", "paged_attn", "delta", "delta_sm100"}

_lib = None


def sources() -> list[Path]:
    return sorted(CSRC.glob("*.cu"))


def _stale(lib: Path, srcs: list[Path]) -> bool:
    if not lib.exists():
        return True
    t = lib.stat().st_mtime
    return any(p.stat().st_mtime > t for p in srcs + list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h")))


def subset_lib(name: str) -> Path:
    return OUT_DIR / f"libkotodama_b200_{name}.so"


def build(force: bool = False, verbose: bool = False, only: Optional[Sequence[str]] = None, name: str = "") -> Path:
    """Compile every ``.cu`` (in parallel) and link the shared library.  No-op when up to date.  ``only``: the sources with
    these stems, linked to the library of the subset ``name``."""
    lib = subset_lib(name) if only else LIB
    srcs = [CSRC / f"{s}.cu" for s in only] if only else sources()
    if not force and not _stale(lib, srcs):
        return lib
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    OBJ_DIR.mkdir(parents=True, exist_ok=True)
    OUT_DIR.mkdir(parents=True, exist_ok=True)

    def compile_one(src: Path) -> Path:
        obj = OBJ_DIR / (src.stem + ".o")
        if not force and not _stale(obj, [src]):
            return obj
        cmd = [nvcc, *NVCC_FLAGS, *([] if src.stem in PRECISE else ["--use_fast_math"]), "-I", str(CSRC), "-c", str(src),
               "-o", str(obj) + ".tmp"]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            print(r.stderr)
        os.replace(str(obj) + ".tmp", obj)
        return obj

    with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 4)) as ex:
        objs = list(ex.map(compile_one, srcs))
    tmp = lib.with_suffix(".so.tmp")
    r = subprocess.run([nvcc, "-shared", "-o", str(tmp), *map(str, objs), "-lcudart_static", "-ldl", "-lrt", "-lpthread"],
                       capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    os.replace(tmp, lib)
    return lib


def use(only: Sequence[str], name: str) -> None:
    """For a process that needs the kernels of these sources alone: loads the full library if it is there and up to
    date, else the subset's, which is compiled first when missing or out of date."""
    global _lib
    if _lib is None:
        path = LIB if not only or not _stale(LIB, sources()) else build(only=only, name=name)
        _lib = ctypes.CDLL(str(path if path.exists() else build()))


def load() -> ctypes.CDLL:
    """Load the library; builds it first when missing and a compiler is available."""
    global _lib
    if _lib is None:
        if not LIB.exists():
            build()
        _lib = ctypes.CDLL(str(LIB))
    return _lib
