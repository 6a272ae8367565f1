"""Builds the CUDA/C++ sources under ``csrc/`` for sm_100a, in-tree, into two libraries:
``libkvb200.so`` (caches, attention, GEMM, collectives of the LitGPT-shaped models) and
``libkvb200_layers.so`` (kernels of models described layer by layer: latent and grouped attention,
state-space recurrence, retention, gated linear attention, gated recurrence, routed experts, token shift, depth averages, norms). Each loads on its own, so a command that needs one
of them compiles no more than that.

Usage: ``python -m keys_values_b200.build_ext [--force] [--verbose]``. nvcc
cross-compiles without a GPU; objects are cached under ``csrc/build`` and only
rebuilt when a source or header is newer.
"""
from __future__ import annotations

import fcntl
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path
from typing import Optional, Sequence

ROOT = Path(__file__).resolve().parent
CSRC = ROOT / "csrc"
BUILD = CSRC / "build"
LIB = ROOT / "libkvb200.so"
LAYERS_LIB = ROOT / "libkvb200_layers.so"
LAYERS_SOURCES = ("gated_linear", "gated_recurrence", "grouped_attn", "latent_attn", "latent_sm100", "layer_edge", "moe", "moe_sm100", "norm_edge", "retention", "ssm", "ssm_sm100")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--expt-relaxed-constexpr", "--expt-extended-lambda", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=default",
]


def _nvcc() -> str:
    cand = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    return cand if os.path.exists(cand) else "nvcc"


def sources(lib: Path = LIB):
    """Sources of one of the two libraries."""
    every = sorted(list(CSRC.glob("*.cu")) + list(CSRC.glob("*.cpp")))
    return [s for s in every if (s.stem in LAYERS_SOURCES) == (lib == LAYERS_LIB)]


def _headers_mtime() -> float:
    hs = list(CSRC.glob("*.h")) + list(CSRC.glob("*.cuh"))
    return max((h.stat().st_mtime for h in hs), default=0.0)


def _compile(src: Path, force: bool, verbose: bool) -> Path:
    obj = BUILD / (src.stem + ".o")
    newest = max(src.stat().st_mtime, _headers_mtime())
    if not force and obj.exists() and obj.stat().st_mtime >= newest:
        return obj
    cmd = [_nvcc(), *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
    if src.suffix == ".cpp":
        cmd = [_nvcc(), *NVCC_FLAGS, "-x", "cu", "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
    if verbose:
        cmd.insert(1, "-Xptxas")
        cmd.insert(2, "-v")
    res = subprocess.run(cmd, capture_output=True, text=True)
    if verbose or res.returncode != 0:
        sys.stderr.write(res.stdout + res.stderr)
    if res.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src.name}")
    return obj


def build(force: bool = False, verbose: bool = False, libs: Optional[Sequence[Path]] = None) -> Path:
    """Compile what is out of date and link ``libs`` (default: both libraries). Returns the path of the first one."""
    libs = [LIB, LAYERS_LIB] if libs is None else list(libs)
    BUILD.mkdir(exist_ok=True)
    with open(BUILD / "lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)  # one process compiles, the others find it done
        srcs = [s for lib in libs for s in sources(lib)]
        with ThreadPoolExecutor(max_workers=min(8, len(srcs))) as ex:
            objs = dict(zip(srcs, ex.map(lambda s: _compile(s, force, verbose), srcs)))
        for lib in libs:
            mine = [objs[s] for s in sources(lib)]
            if force or not lib.exists() or any(o.stat().st_mtime > lib.stat().st_mtime for o in mine):
                part = lib.with_suffix(".so.part")
                res = subprocess.run([_nvcc(), "-shared", "-o", str(part), *map(str, mine), "-lcudart"], capture_output=True, text=True)
                if res.returncode != 0:
                    sys.stderr.write(res.stdout + res.stderr)
                    raise RuntimeError(f"link of {lib.name} failed")
                os.replace(part, lib)
    return libs[0]


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
