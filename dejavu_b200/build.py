"""Builds the C-ABI libraries of sm_100a kernels in-tree with nvcc.

    python -m dejavu_b200.build [--force] [--verbose] [--lib sparse|hybrid|routed]

  sparse  libdejavu_b200.so         the contextual-sparse OPT decode path
  hybrid  libdejavu_b200_hybrid.so  gated linear attention, sliding-window attention, hyper-connected streams
  routed  libdejavu_b200_routed.so  matrix memories, latent attention, routed feed-forwards

Each .cu file is compiled to an object in parallel, then linked into the shared libraries that sit next to this file.
Nothing is cached outside the package directory. A library can be built alone, so that a program that serves one kind
of model compiles only what it needs.
"""
from __future__ import annotations

import argparse
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
OBJ = PKG / "build"
LIB = PKG / "libdejavu_b200.so"
HYBRID_LIB = PKG / "libdejavu_b200_hybrid.so"
ROUTED_LIB = PKG / "libdejavu_b200_routed.so"
LIBS = {"sparse": LIB, "hybrid": HYBRID_LIB, "routed": ROUTED_LIB}

# translation units of the hybrid decoders' libraries; those both use are compiled once and linked into both
_BOTH = ("api", "hybrid_gemv", "hybrid_residual", "hybrid_rotary", "hybrid_window_simple", "hybrid_window_prefill")
_UNITS = {"hybrid": _BOTH + ("hybrid_attention", "hybrid_gla", "hybrid_gla_mma"),
          "routed": _BOTH + ("hybrid_mlstm", "hybrid_mlstm_prefill", "hybrid_latent", "hybrid_latent_decode", "hybrid_moe",
                             "hybrid_moe_gemm")}

NVCC_FLAGS = [
    "-O3",
    "-std=c++17",
    "-gencode",
    "arch=compute_100a,code=sm_100a",
    "-lineinfo",
    "-Xcompiler",
    "-fPIC",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found; set NVCC=/path/to/nvcc")


def sources(lib: str | None = None) -> list[Path]:
    """Translation units of a library (of all, without a name). api.cu, the plumbing, is part of each."""
    out = sorted(CSRC.glob("*.cu"))
    if lib is None:
        return out
    if lib in _UNITS:
        return [p for p in out if p.stem in _UNITS[lib]]
    return [p for p in out if not p.stem.startswith("hybrid_")]


def _stale(target: Path, deps: list[Path]) -> bool:
    if not target.exists():
        return True
    t = target.stat().st_mtime
    return any(d.stat().st_mtime > t for d in deps)


def build(force: bool = False, verbose: bool = False, libs: tuple[str, ...] = tuple(LIBS)) -> Path:
    """Compiles what is stale of the named libraries and returns the path of the first one. DJV_NVCC_FLAGS in the
    environment adds flags (e.g. -DDJV_RING_TRACE for the phase stamps of the one-pass MLP kernel; use --force, the
    flag is not part of the staleness check)."""
    nvcc = _nvcc()
    extra = os.environ.get("DJV_NVCC_FLAGS", "").split()
    OBJ.mkdir(exist_ok=True)
    headers = sorted(CSRC.glob("*.cuh")) + sorted((PKG.parent / "include").glob("*.h"))
    wanted = sorted({src for lib in libs for src in sources(lib)})
    jobs = []
    for src in wanted:
        obj = OBJ / (src.stem + ".o")
        if force or _stale(obj, [src] + headers):
            cmd = [nvcc, *NVCC_FLAGS, *extra, "-c", str(src), "-o", str(obj)]
            if verbose:
                cmd.insert(1, "-Xptxas")
                cmd.insert(2, "-v")
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        return cmd, r

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        for cmd, r in ex.map(run, jobs):
            if verbose or r.returncode != 0:
                sys.stderr.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
            if r.returncode != 0:
                raise RuntimeError(f"nvcc failed on {cmd[-3]}")
    for lib in libs:
        objs = [OBJ / (s.stem + ".o") for s in sources(lib)]
        if force or _stale(LIBS[lib], objs):
            part = LIBS[lib].with_suffix(f".{os.getpid()}.tmp")
            cmd = [nvcc, "-shared", "-o", str(part), *map(str, objs), "-Xcompiler", "-fPIC", "-lcudart"]
            r = subprocess.run(cmd, capture_output=True, text=True)
            if r.returncode != 0:
                sys.stderr.write(r.stdout + r.stderr)
                raise RuntimeError("link failed")
            os.replace(part, LIBS[lib])
    return LIBS[libs[0]]


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true", help="print ptxas register / shared-memory usage")
    ap.add_argument("--lib", choices=sorted(LIBS), help="build this library only")
    a = ap.parse_args()
    names = (a.lib,) if a.lib else tuple(LIBS)
    build(force=a.force, verbose=a.verbose, libs=names)
    for name in names:
        print(LIBS[name])
