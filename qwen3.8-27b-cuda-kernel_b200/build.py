"""In-tree build of the native libraries (no GPU needed: nvcc cross-compiles for sm_100a).

    python qwen3.8-27b-cuda-kernel_b200/build.py [--force] [--verbose] [--family NAME]

Outputs, next to this file:
    lib/libq38_kernels.so   every CUDA kernel + the C ABI declared in include/q38_kernels.h
    lib/libq38_engine.so    the C++20 host engine (ModelFile, KvCache, ModelRunner, Engine) + its C ABI

The sources belong to model families (FAMILIES) or are shared. A build of one family only (`build(family=...)`) compiles
its own and the shared sources and puts the same two libraries into lib/<family>/: an engine that serves that family's
architectures and nothing else.
"""

from __future__ import annotations

import argparse
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

HERE = Path(__file__).resolve().parent
ROOT = HERE.parent
CSRC = HERE / "csrc"
HOST = HERE / "host"
OBJ = HERE / "build"
LIB = HERE / "lib"

NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
CUDA_LIB = str(Path(NVCC).resolve().parents[1] / "lib64")
CUDA_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++20", "-Xcompiler", "-fPIC",
              "--expt-relaxed-constexpr", "-I", str(ROOT / "include")]
HOST_FLAGS = ["-std=c++20", "-O2", "-fPIC", "-I", str(ROOT / "include"), "-I", str(HOST / "include"),
              "-I", "/usr/local/cuda/include"]


# sources of one model family; everything else is shared
FAMILIES = {
    "bq": {"cu": {"attention", "gdn", "qgemm", "qgemm_stream", "qgemm_umma"}, "host": {"bq_model"}},
    "layer_list": {"cu": {"dense_gemm", "dense_umma", "mixed_attention", "mixed_attention_mma", "recurrent", "row_norm",
                          "stream_norm", "retention", "latent_attention", "packed_attention"},
                   "host": {"layer_list_model", "fegenex", "nololix"}},
}
ARCHITECTURE_FAMILY = {"Qwen3.8": "bq", "Fegenex": "layer_list", "Nololix": "layer_list"}


def _stale(target: Path, deps: list[Path]) -> bool:
    if not target.exists():
        return True
    t = target.stat().st_mtime
    return any(d.stat().st_mtime > t for d in deps)


def _run(cmd: list[str], verbose: bool) -> None:
    if verbose:
        print("+", " ".join(cmd), flush=True)
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        sys.stderr.write(r.stdout + r.stderr)
        raise RuntimeError("build step failed: " + " ".join(cmd))
    if verbose and (r.stdout or r.stderr):
        print(r.stdout + r.stderr)


def _sources(folder: Path, pattern: str, kind: str, family: str | None) -> list[Path]:
    skip = set().union(*(f[kind] for name, f in FAMILIES.items() if family is not None and name != family))
    return [p for p in sorted(folder.glob(pattern)) if p.stem not in skip]


def build(force: bool = False, verbose: bool = False, ptxas_verbose: bool = False,
          family: str | None = None) -> dict[str, Path]:
    lib_dir = LIB if family is None else LIB / family
    OBJ.mkdir(exist_ok=True)
    lib_dir.mkdir(parents=True, exist_ok=True)
    cu_headers = sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h")) + [ROOT / "include" / "q38_kernels.h"]
    jobs = []
    cu_objs = []
    for src in _sources(CSRC, "*.cu", "cu", family):
        obj = OBJ / (src.stem + ".o")
        cu_objs.append(obj)
        if force or _stale(obj, [src] + cu_headers):
            extra = ["-Xptxas", "-v"] if ptxas_verbose else []
            jobs.append([NVCC, *CUDA_FLAGS, *extra, "-c", str(src), "-o", str(obj)])
    host_headers = sorted((HOST / "include").rglob("*.h")) + sorted((HOST / "src").glob("*.h")) + sorted((ROOT / "include").glob("*.h"))
    host_objs = []
    for src in _sources(HOST / "src", "*.cpp", "host", family):
        obj = OBJ / ("host_" + src.stem + ".o")
        host_objs.append(obj)
        if force or _stale(obj, [src] + host_headers):
            jobs.append(["g++", *HOST_FLAGS, "-c", str(src), "-o", str(obj)])
    jobs.sort(key=lambda c: c[0] != NVCC)  # the long ones first
    with ThreadPoolExecutor(max_workers=os.cpu_count() or 4) as pool:
        list(pool.map(lambda c: _run(c, verbose or ptxas_verbose), jobs))
    kernels_so = lib_dir / "libq38_kernels.so"
    if force or _stale(kernels_so, cu_objs):
        # both libraries use the one shared CUDA runtime of the process (a host application's, or torch's in the
        # tests and benchmarks): same soname, so whichever copy is loaded first serves everybody
        _run([NVCC, "-shared", "--cudart", "shared", "-o", str(kernels_so), *map(str, cu_objs),
              "-Xlinker", f"-rpath,{CUDA_LIB}"], verbose)
    out = {"kernels": kernels_so}
    if host_objs:
        engine_so = lib_dir / "libq38_engine.so"
        if force or _stale(engine_so, host_objs + [kernels_so]):
            _run(["g++", "-shared", "-o", str(engine_so), *map(str, host_objs), "-L", str(lib_dir), "-lq38_kernels",
                  f"-L{CUDA_LIB}", "-lcudart", "-ldl", "-lrt", "-lpthread",
                  f"-Wl,-rpath,$ORIGIN:{CUDA_LIB}"], verbose)
        out["engine"] = engine_so
    return out


def up_to_date(family: str | None) -> bool:
    """Whether the libraries of this build exist and are newer than all their sources."""
    lib_dir = LIB if family is None else LIB / family
    deps = (_sources(CSRC, "*.cu", "cu", family) + list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h")) +
            _sources(HOST / "src", "*.cpp", "host", family) + list((HOST / "src").glob("*.h")) +
            list((HOST / "include").rglob("*.h")) + list((ROOT / "include").glob("*.h")))
    return not any(_stale(lib_dir / n, deps) for n in ("libq38_kernels.so", "libq38_engine.so"))


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    ap.add_argument("--ptxas", action="store_true", help="print registers / spills / shared memory per kernel")
    ap.add_argument("--family", choices=sorted(FAMILIES), help="this model family only, into lib/<family>/")
    a = ap.parse_args()
    for name, path in build(a.force, a.verbose, a.ptxas, a.family).items():
        print(f"{name}: {path}")
