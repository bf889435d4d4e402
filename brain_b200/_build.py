"""In-tree native build: every ``csrc/**/*.cu`` is compiled by nvcc for sm_100a into one shared
library (``brain_b200/_lib/libbrain_b200.so``, C ABI, loaded with ctypes) and the host runtime
(``csrc/**/*.cpp``) into ``brain_b200/_lib/libbrain_host.so``.

Nothing here needs a GPU: nvcc cross-compiles.  Objects are rebuilt only when their source (or a
header) is newer, so repeated calls are cheap.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parent.parent
CSRC = ROOT / "csrc"
LIBDIR = Path(__file__).resolve().parent / "_lib"
OBJDIR = ROOT / "build" / "obj"

CUDA_LIB = LIBDIR / "libbrain_b200.so"
HOST_LIB = LIBDIR / "libbrain_host.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--use_fast_math", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
    "--expt-relaxed-constexpr", "-Xptxas", "-v",
]
#: translation units whose arithmetic feeds the optimiser state or the loss: compiled without
#: --use_fast_math (IEEE division and square root in the AdamW update, exact exp/log in the CE)
#: (the hybrid decoder's norms, recurrence and fp32 path: what is computed in 32-bit keeps its 32 bits)
EXACT_MATH = {"adamw.cu", "rs_adamw.cu", "ce.cu", "hybrid_rows.cu", "mamba2.cu", "attn_rows.cu", "sgemm.cu",
              "depth_rows.cu", "latent_rows.cu", "delta.cu", "rglru.cu", "mlstm.cu", "experts.cu",
              "stream_rows.cu", "head_rows.cu", "linear_state.cu", "gla_tcgen05.cu"}
CXX_FLAGS = ["-O3", "-std=c++17", "-fPIC", "-fvisibility=hidden", "-pthread", "-march=x86-64-v3"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found")


def _newest_header() -> float:
    hs = list(CSRC.rglob("*.cuh")) + list(CSRC.rglob("*.hpp")) + list(CSRC.rglob("*.h"))
    return max((h.stat().st_mtime for h in hs), default=0.0)


def _stale(src: Path, obj: Path, hdr_mtime: float) -> bool:
    if not obj.exists():
        return True
    m = obj.stat().st_mtime
    return src.stat().st_mtime > m or hdr_mtime > m


def _run(cmd: list[str], log: Path | None = None) -> None:
    p = subprocess.run(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if log is not None:
        log.write_text(p.stdout)
    if p.returncode != 0:
        sys.stderr.write(p.stdout)
        raise RuntimeError("build failed: " + " ".join(cmd))


def build_cuda(force: bool = False, verbose: bool = False) -> Path:
    return _build_cuda(sorted(CSRC.rglob("*.cu")), CUDA_LIB, force, verbose)


def _build_cuda(srcs, lib: Path, force: bool = False, verbose: bool = False) -> Path:
    OBJDIR.mkdir(parents=True, exist_ok=True)
    LIBDIR.mkdir(parents=True, exist_ok=True)
    hdr = _newest_header()
    nvcc = _nvcc()
    jobs = []
    objs = []
    for s in srcs:
        o = OBJDIR / (str(s.relative_to(CSRC)).replace("/", "__") + ".o")
        objs.append(o)
        if force or _stale(s, o, hdr):
            jobs.append((s, o))

    def compile_one(so):
        s, o = so
        extra = ["-DBB_TIMELINE"] if os.environ.get("BB_TIMELINE") == "1" else []
        flags = NVCC_FLAGS
        if s.name in EXACT_MATH:
            flags = [f for f in NVCC_FLAGS if f != "--use_fast_math"]
        _run([nvcc, *flags, *extra, "-I", str(CSRC), "-c", str(s), "-o", str(o)],
             log=o.with_suffix(".log"))
        if verbose:
            print(f"[build] {s.relative_to(ROOT)}")

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 4)) as ex:
            list(ex.map(compile_one, jobs))
    if jobs or not lib.exists() or any(o.stat().st_mtime > lib.stat().st_mtime for o in objs):
        # linked beside its place and moved there, so a library that another process has open stays whole
        tmp = lib.with_suffix(f".{os.getpid()}.tmp")
        _run([nvcc, "-shared", "-o", str(tmp), *map(str, objs), "-lcudart"])
        os.replace(tmp, lib)
    return lib


def build_host(force: bool = False, verbose: bool = False) -> Path:
    return _build_host(sorted(CSRC.rglob("*.cpp")), HOST_LIB, force, verbose)


def _build_host(srcs, lib: Path, force: bool = False, verbose: bool = False) -> Path:
    OBJDIR.mkdir(parents=True, exist_ok=True)
    LIBDIR.mkdir(parents=True, exist_ok=True)
    hdr = _newest_header()
    cxx = os.environ.get("CXX", "g++")
    jobs, objs = [], []
    for s in srcs:
        o = OBJDIR / (str(s.relative_to(CSRC)).replace("/", "__") + ".o")
        objs.append(o)
        if force or _stale(s, o, hdr):
            jobs.append((s, o))

    def compile_one(so):
        s, o = so
        _run([cxx, *CXX_FLAGS, "-I", str(CSRC), "-c", str(s), "-o", str(o)])
        if verbose:
            print(f"[build] {s.relative_to(ROOT)}")

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 4)) as ex:
            list(ex.map(compile_one, jobs))
    if jobs or not lib.exists() or any(o.stat().st_mtime > lib.stat().st_mtime for o in objs):
        tmp = lib.with_suffix(f".{os.getpid()}.tmp")
        _run([cxx, "-shared", "-o", str(tmp), *map(str, objs), "-pthread"])
        os.replace(tmp, lib)
    return lib


#: translation units of the bounds-checking library (kernels whose addresses depend on data) and
#: what they need at link time
BOUNDS_TUS = ["kernels/elementwise.cu", "kernels/ce.cu", "kernels/moe.cu", "common/host.cu"]
BOUNDS_LIB = LIBDIR / "libbrain_b200_bounds.so"


def build_bounds(force: bool = False, verbose: bool = False) -> Path:
    """A second, small library of the index-driven kernels compiled with -DBB_DEBUG_BOUNDS: every
    data-dependent index is checked against its extent, a violation writes an error code and skips
    the access.  Loaded by tests only: production code never links it."""
    OBJDIR.mkdir(parents=True, exist_ok=True)
    LIBDIR.mkdir(parents=True, exist_ok=True)
    hdr = _newest_header()
    nvcc = _nvcc()
    objs, jobs = [], []
    for rel in BOUNDS_TUS:
        s = CSRC / rel
        o = OBJDIR / ("bounds__" + rel.replace("/", "__") + ".o")
        objs.append(o)
        if force or _stale(s, o, hdr):
            jobs.append((s, o))
    for s, o in jobs:
        flags = [f for f in NVCC_FLAGS if f != "--use_fast_math"] if s.name in EXACT_MATH else NVCC_FLAGS
        _run([nvcc, *flags, "-DBB_DEBUG_BOUNDS", "-I", str(CSRC), "-c", str(s), "-o", str(o)],
             log=o.with_suffix(".log"))
        if verbose:
            print(f"[build] bounds {s.relative_to(ROOT)}")
    if jobs or not BOUNDS_LIB.exists():
        _run([nvcc, "-shared", "-o", str(BOUNDS_LIB), *map(str, objs), "-lcudart"])
    return BOUNDS_LIB


#: what serving a hybrid decoder needs of the kernel library, for programs that compile on first use
HYBRID_TUS = ["common/host.cu", "kernels/attn_rows.cu", "kernels/delta.cu", "kernels/depth_rows.cu", "kernels/experts.cu",
              "kernels/flash_fwd.cu",
              "kernels/gemm_2cta.cu", "kernels/gemm_groups.cu", "kernels/gemm_tcgen05.cu", "kernels/gla_tcgen05.cu", "kernels/head_rows.cu",
              "kernels/hybrid_rows.cu",
              "kernels/latent_decode.cu", "kernels/latent_rows.cu", "kernels/linear_state.cu",
              "kernels/mamba2.cu", "kernels/mlstm.cu", "kernels/paged_kv.cu",
              "kernels/rglru.cu",
              "kernels/router_quant_sample.cu", "kernels/sgemm.cu", "kernels/ssd_tcgen05.cu",
              "kernels/stream_rows.cu", "serve/hybrid_forward.cu"]
HYBRID_LIB = LIBDIR / "libbrain_b200_hybrid.so"
#: ... and of the host runtime (checkpoint reader, pages, slots, scheduler)
HYBRID_HOST_SRCS = ["runtime/data.cpp", "runtime/safetensors.cpp", "runtime/serving.cpp"]
HYBRID_HOST_LIB = LIBDIR / "libbrain_host_hybrid.so"


def build_hybrid(verbose: bool = False) -> Path:
    """The kernel library reduced to :data:`HYBRID_TUS` (objects are shared with the full build)."""
    return _build_cuda([CSRC / t for t in HYBRID_TUS], HYBRID_LIB, verbose=verbose)


def build_hybrid_host(verbose: bool = False) -> Path:
    return _build_host([CSRC / t for t in HYBRID_HOST_SRCS], HYBRID_HOST_LIB, verbose=verbose)


def library_current(lib: Path, suffix: str) -> bool:
    """The library exists and is newer than every source file with that suffix and every header."""
    if not lib.exists():
        return False
    m = lib.stat().st_mtime
    return _newest_header() <= m and all(s.stat().st_mtime <= m for s in CSRC.rglob("*" + suffix))


def build_all(force: bool = False, verbose: bool = False) -> None:
    build_host(force, verbose)
    build_cuda(force, verbose)
    build_bounds(force, verbose)


def ptxas_report() -> str:
    """Concatenated ``-Xptxas -v`` output of the last build (registers, spills, smem per kernel)."""
    out = []
    for log in sorted(OBJDIR.glob("*.log")):
        out.append(f"== {log.name}\n{log.read_text()}")
    return "\n".join(out)


if __name__ == "__main__":
    build_all(force="--force" in sys.argv, verbose=True)
    if "--report" in sys.argv:
        print(ptxas_report())
