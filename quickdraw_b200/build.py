"""Build the C-ABI CUDA libraries in-tree: ``python -m quickdraw_b200.build [nvfp4|hybrid|recurrent|latent ...]``.

Plain nvcc, shared objects for sm_100a only, no link against libtorch: the host side passes raw
device pointers through ctypes.  Several libraries, so that a model only needs its own kernels
compiled: ``libquickdraw_b200.so`` (NVFP4 / FP8 models), ``libquickdraw_b200_hybrid.so`` (what all
bf16-weight models use) and one for each family of mixers that only some of those have,
``_recurrent`` (gated linear recurrences) and ``_latent`` (latent attention).  Without a name all
are built.
"""

from __future__ import annotations

import os
import subprocess
import sys
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
LIB = PKG / "libquickdraw_b200.so"
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-lineinfo", "-std=c++17",
         "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr"]

COMMON = ("library",)
HYBRID_SOURCES = {"hybrid": ("linear", "residual", "window_attention"), "recurrent": ("linear_recurrence",),
                  "latent": ("latent_attention",)}
HYBRID_HEADERS = ("common.cuh", "typed.cuh", "softmax_attention.cuh")
TARGETS = ("nvfp4", *HYBRID_SOURCES)


def sources(target: str) -> list[Path]:
    if target in HYBRID_SOURCES:
        return [CSRC / f"{name}.cu" for name in COMMON + HYBRID_SOURCES[target]]
    others = {name for names in HYBRID_SOURCES.values() for name in names}
    return [path for path in sorted(CSRC.glob("*.cu")) if path.stem not in others]


def library(target: str) -> Path:
    return LIB if target == "nvfp4" else PKG / f"libquickdraw_b200_{target}.so"


def stale(target: str = "nvfp4") -> bool:
    lib = library(target)
    if not lib.exists():
        return True
    headers = ([CSRC / name for name in HYBRID_HEADERS] if target in HYBRID_SOURCES else sorted(CSRC.glob("*.cuh")))
    headers += sorted((PKG.parent / "include").glob("*.h"))
    return max(p.stat().st_mtime for p in sources(target) + headers) > lib.stat().st_mtime


def build(force: bool = False, verbose: bool = False, targets=TARGETS) -> list[Path]:
    """Compile what is out of date; every source of every requested library in parallel."""
    wanted = [t for t in targets if force or stale(t)]
    build_dir = PKG / "build"
    build_dir.mkdir(exist_ok=True)
    procs, objects = [], {t: [build_dir / (src.stem + ".o") for src in sources(t)] for t in wanted}
    for src in dict.fromkeys(src for t in wanted for src in sources(t)):
        cmd = [NVCC, *FLAGS, "-c", str(src), "-o", str(build_dir / (src.stem + ".o"))]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for src, proc in procs:
        out, _ = proc.communicate()
        if proc.returncode != 0 or verbose:
            sys.stderr.write(f"== {src.name}\n{out}\n")
        failed |= proc.returncode != 0
    if failed:
        raise RuntimeError("nvcc failed")
    for t in wanted:
        subprocess.run([NVCC, "-shared", "-o", str(library(t)), *map(str, objects[t]), "-lcudart"], check=True)
    return [library(t) for t in targets]


if __name__ == "__main__":
    names = [a for a in sys.argv[1:] if not a.startswith("-")] or list(TARGETS)
    print(*build(force="--force" in sys.argv, verbose="-v" in sys.argv, targets=names), sep="\n")
