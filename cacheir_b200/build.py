"""Build the CUDA libraries in-tree with nvcc for sm_100a.

Usage: python -m cacheir_b200.build [--force] [--verbose] [--group NAME]

Plain C-ABI shared objects (no torch, no pybind), each a group of the .cu files
under csrc/ compiled with -gencode arch=compute_100a,code=sm_100a and linked
with the static CUDA runtime: `core` (libcacheir_b200.so, Llama-shaped models),
`ragged` (dense products and row operators of the families with ragged steps),
`hybrid` (latent attention), `recurrence` (linear recurrences, matrix memory, state
spaces), `experts` (tied attention, mixtures of experts), `talking` (talking-heads
attention) and `delta` (short convolutions, delta rule). A model family names the groups it needs, so a fresh
checkout compiles only those. Objects are rebuilt only when their source or a
header is newer.
"""
from __future__ import annotations

import argparse
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG_DIR = Path(__file__).resolve().parent
CSRC = PKG_DIR / "csrc"
INCLUDE = PKG_DIR.parent / "include"
BUILD_DIR = PKG_DIR / "build"
LIB_DIR = PKG_DIR / "lib"
SHARED = ("glue", "misc")            # in the core and the ragged library: argmax, position bookkeeping, error text
GROUP_FILES = {
    "ragged": ("dense_gemm", "hybrid_glue") + SHARED,
    "hybrid": ("latent_attention",),
    "recurrence": ("linear_recurrence",),
    "talking": ("talking_attention", "talking_prompt"),
    "delta": ("short_conv", "delta_rule"),
    "experts": ("tied_attention", "tied_prompt", "grouped_gemm", "expert_routing"),
}
LIB_PATHS = {"core": LIB_DIR / "libcacheir_b200.so", **{name: LIB_DIR / f"libcacheir_b200_{name}.so" for name in GROUP_FILES}}
LIB_PATH = LIB_PATHS["core"]

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]


def find_nvcc() -> str:
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not Path(nvcc).exists():
        raise RuntimeError("nvcc not found; cacheir_b200 needs the CUDA toolkit to build its kernels")
    return nvcc


def _stale(target: Path, deps: list[Path]) -> bool:
    if not target.exists():
        return True
    mtime = target.stat().st_mtime
    return any(dep.stat().st_mtime > mtime for dep in deps)


def group_sources(group: str) -> list[Path]:
    if group in GROUP_FILES:
        return sorted(CSRC / f"{name}.cu" for name in GROUP_FILES[group])
    others = {name for names in GROUP_FILES.values() for name in names} - set(SHARED)
    return sorted(src for src in CSRC.glob("*.cu") if src.stem not in others)


def build(force: bool = False, verbose: bool = False, groups: tuple[str, ...] = tuple(LIB_PATHS)) -> Path:
    """Bring the libraries of `groups` up to date; returns the path of the first one."""
    nvcc = find_nvcc()
    BUILD_DIR.mkdir(parents=True, exist_ok=True)
    LIB_DIR.mkdir(parents=True, exist_ok=True)
    sources = sorted({src for group in groups for src in group_sources(group)})
    headers = sorted(CSRC.glob("*.cuh")) + sorted(INCLUDE.glob("*.h")) + [Path(__file__)]
    extra = ["-Xptxas", "-v"] if verbose else []

    def compile_one(src: Path) -> Path:
        obj = BUILD_DIR / (src.stem + ".o")
        if force or _stale(obj, [src] + headers):
            cmd = [nvcc, *NVCC_FLAGS, *extra, "-I", str(INCLUDE), "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
            proc = subprocess.run(cmd, capture_output=True, text=True)
            if verbose or proc.returncode != 0:
                sys.stderr.write(proc.stdout + proc.stderr)
            if proc.returncode != 0:
                raise RuntimeError(f"nvcc failed on {src.name}")
        return obj

    with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 1)) as pool:
        objects = dict(zip(sources, pool.map(compile_one, sources)))

    for group in groups:
        target, members = LIB_PATHS[group], [objects[src] for src in group_sources(group)]
        if force or _stale(target, members):
            part = target.with_suffix(".so.part")      # a reader never sees a half-written library
            cmd = [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-cudart", "static",
                   "-o", str(part), *map(str, members)]
            proc = subprocess.run(cmd, capture_output=True, text=True)
            if proc.returncode != 0:
                sys.stderr.write(proc.stdout + proc.stderr)
                raise RuntimeError(f"linking {target.name} failed")
            os.replace(part, target)
    return LIB_PATHS[groups[0]]


if __name__ == "__main__":
    parser = argparse.ArgumentParser(description=__doc__)
    parser.add_argument("--force", action="store_true")
    parser.add_argument("--verbose", action="store_true", help="print ptxas register/smem usage")
    parser.add_argument("--group", choices=sorted(LIB_PATHS), help="build one library only")
    args = parser.parse_args()
    for name in (args.group,) if args.group else tuple(LIB_PATHS):
        print(build(force=args.force, verbose=args.verbose, groups=(name,)))
