"""In-tree build of the CUDA kernel library for sm_100a.

``python -m mindspeed_rl_b200.csrc.build`` compiles every ``*.cu`` under this directory
with ``nvcc -gencode arch=compute_100a,code=sm_100a -lineinfo`` into objects and links them
into ``mindspeed_rl_b200/_C/libmsrl_b200.so`` (plain ``extern "C"`` entry points, loaded with
ctypes -- no Python or torch headers involved, so a full rebuild takes seconds).  C++-only
sources (``*.cpp``: block manager, host runtime helpers) are compiled with g++ into the same
library.  Objects are rebuilt only when their source or a header is newer.
"""
from __future__ import annotations

import concurrent.futures as cf
import os
import shutil
import subprocess
import sys
from pathlib import Path
from typing import List

CSRC = Path(__file__).resolve().parent
PKG = CSRC.parent
OUT_DIR = PKG / "_C"
OBJ_DIR = OUT_DIR / "obj"
LIB_PATH = OUT_DIR / "libmsrl_b200.so"
HOST_LIB_PATH = OUT_DIR / "libmsrl_host.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--use_fast_math", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
    "--expt-relaxed-constexpr", "-Xptxas", "-v",
]
# kernels whose results are specified in 32-bit (an fp32 residual, recurrent state, fp32 attention): compiled
# without the approximate divisions, square roots, exponentials and flush-to-zero of --use_fast_math
PRECISE = {"residual_stream", "delta_rule", "latent_attention", "latent_decode_tcgen05", "grouped_gemm_simt",
           "matrix_memory", "matrix_memory_tcgen05", "qkv_prep", "conv_qkv", "attention_simt",
           "moe", "wkv", "wkv_chunk", "min_gru"}
CXX_FLAGS = ["-O2", "-std=c++17", "-fPIC", "-fvisibility=hidden", "-pthread"]


# kernels of one model family, linked into a library of their own (``_C/libmsrl_<group>.so``): a process that serves the
# family from a fresh checkout compiles these and nothing else (the forward of the family, without the sampler)
_STREAM = ("residual_stream", "grouped_gemm_simt", "moe", "moe_gemm_tcgen05", "attention", "attention_tcgen05", "attention_simt",
           "paged_rows", "gemm2cta_tcgen05")
GROUPS = {
    "pumotar": (*_STREAM, "delta_rule", "latent_attention", "latent_decode_tcgen05"),
    "gapevik": (*_STREAM, "delta_rule", "latent_attention", "latent_decode_tcgen05", "conv_qkv", "decode", "decode_prefix_tcgen05"),
    "lunelorn": (*_STREAM, "matrix_memory", "matrix_memory_tcgen05", "qkv_prep", "wkv", "wkv_chunk", "min_gru", "decode",
                 "decode_prefix_tcgen05"),
    "sunatar": (*_STREAM, "matrix_memory", "matrix_memory_tcgen05", "qkv_prep", "decode", "decode_prefix_tcgen05"),
}


def group_path(name: str) -> Path:
    return OUT_DIR / f"libmsrl_{name}.so"


def _nvcc() -> str:
    cand = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(cand):
        raise RuntimeError("nvcc not found; the CUDA kernels cannot be built")
    return cand


def _newest_header() -> float:
    hs = list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h")) + list(CSRC.glob("*.hpp"))
    return max((h.stat().st_mtime for h in hs), default=0.0)


def _compile_one(src: Path, force: bool, log_dir: Path) -> Path:
    obj = OBJ_DIR / (src.stem + ".o")
    stamp = max(src.stat().st_mtime, _newest_header(), Path(__file__).stat().st_mtime)
    if not force and obj.exists() and obj.stat().st_mtime >= stamp:
        return obj
    if src.suffix == ".cu":
        flags = [f for f in NVCC_FLAGS if f != "--use_fast_math" or src.stem not in PRECISE]
        cmd = [_nvcc(), *flags, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
    else:
        cmd = ["g++", *CXX_FLAGS, "-I", str(CSRC), "-I", "/usr/local/cuda/include", "-c", str(src),
               "-o", str(obj)]
    res = subprocess.run(cmd, capture_output=True, text=True)
    (log_dir / (src.stem + ".log")).write_text(res.stdout + res.stderr)
    if res.returncode != 0:
        raise RuntimeError(f"compilation of {src.name} failed:\n{res.stdout}\n{res.stderr}")
    return obj


def sources() -> List[Path]:
    return sorted(CSRC.glob("*.cu")) + sorted(CSRC.glob("*.cpp"))


def _stale(lib: Path, deps: List[Path], force: bool = False) -> bool:
    return force or not lib.exists() or any(o.stat().st_mtime > lib.stat().st_mtime for o in deps)


def _link(lib: Path, objs: List[Path], cuda: bool) -> None:
    # linked beside its place and moved there: a process that finds the library finds a whole one
    tmp = lib.with_name(f"{lib.name}.{os.getpid()}")
    if cuda:
        cmd = [_nvcc(), "-shared", "-o", str(tmp), *map(str, objs), "-gencode", "arch=compute_100a,code=sm_100a",
               "-cudart", "static", "-Xcompiler", "-fPIC", "-Xlinker", "-z,noexecstack"]
    else:
        cmd = ["g++", "-shared", "-o", str(tmp), *map(str, objs), "-pthread"]
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"link of {lib.name} failed:\n{res.stdout}\n{res.stderr}")
    os.replace(tmp, lib)


def _compile_all(srcs: List[Path], force: bool) -> List[Path]:
    OBJ_DIR.mkdir(parents=True, exist_ok=True)
    log_dir = OUT_DIR / "logs"
    log_dir.mkdir(exist_ok=True)
    with cf.ThreadPoolExecutor(max_workers=min(8, len(srcs) or 1)) as pool:
        return list(pool.map(lambda s: _compile_one(s, force, log_dir), srcs))


def build_group(name: str) -> Path:
    """Compile and link one group's kernels and the host-only library."""
    cu = [CSRC / f"{stem}.cu" for stem in GROUPS[name]]
    host = sorted(CSRC.glob("*.cpp"))
    objs = _compile_all(cu + host, force=False)
    lib = group_path(name)
    if _stale(lib, objs[:len(cu)]):
        _link(lib, objs[:len(cu)], cuda=True)
    if host and _stale(HOST_LIB_PATH, objs[len(cu):]):
        _link(HOST_LIB_PATH, objs[len(cu):], cuda=False)
    return lib


def build(force: bool = False, verbose: bool = False) -> Path:
    srcs = sources()
    objs = _compile_all(srcs, force)
    cu_objs = [o for s, o in zip(srcs, objs) if s.suffix == ".cu"]
    host_objs = [o for s, o in zip(srcs, objs) if s.suffix == ".cpp"]
    if cu_objs and _stale(LIB_PATH, cu_objs, force):
        _link(LIB_PATH, cu_objs, cuda=True)
    if host_objs and _stale(HOST_LIB_PATH, host_objs, force):
        # host-only runtime pieces (block manager, ...) load on machines without CUDA
        _link(HOST_LIB_PATH, host_objs, cuda=False)
    if verbose:
        for s in srcs:
            log = OUT_DIR / "logs" / (s.stem + ".log")
            if log.exists():
                sys.stdout.write(f"== {s.name}\n{log.read_text()}\n")
    return LIB_PATH


if __name__ == "__main__":
    p = build(force="--force" in sys.argv, verbose="-v" in sys.argv)
    print(p)
