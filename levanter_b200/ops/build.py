"""In-tree build of the sm_100a kernel library.

All CUDA sources under ``csrc/`` are compiled by ``nvcc`` for
``arch=compute_100a,code=sm_100a`` and linked into one shared object,
``_lib/liblevanter_b200.so``, which :mod:`levanter_b200.ops.lib` loads with
``ctypes``.  The kernels expose plain ``extern "C"`` launchers (raw pointers +
stream), so nothing here depends on the PyTorch C++ headers and a full
rebuild takes seconds.  nvcc cross-compiles without a GPU.
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

CSRC = Path(__file__).resolve().parent / "csrc"
LIBDIR = Path(__file__).resolve().parent / "_lib"
LIBNAME = "liblevanter_b200.so"

# What a process that only serves a model needs (``lib.use_serving_library``): a subset of the same objects in a library of its
# own, so that the first run in a fresh checkout compiles these sources and no others.
SERVING_LIBNAME = "liblevanter_b200_serving.so"
SERVING_SOURCES = ("attention_any", "depth_stream", "elementwise", "flash_attn_fwd2", "gated_scan", "gemm_bf16", "gemm_pair", "gemm_skinny",
                   "linear_attention", "linear_attention_umma", "moe_experts", "page_table", "paged_attention", "paged_latent", "qkv_prep",
                   "residual_stream", "sampler")

# Kernels whose results are 32-bit throughout (norms of an fp32 stream, router scores, rotary angles, recurrences, fp32 attention): no
# fast-math exponentials, divisions or square roots.
ACCURATE_SOURCES = ("attention_any", "depth_stream", "gated_scan", "linear_attention", "linear_attention_umma", "moe_experts", "qkv_prep",
                    "residual_stream")

NVCC_FLAGS = [
    "-gencode",
    "arch=compute_100a,code=sm_100a",
    "-lineinfo",
    "-O3",
    "-std=c++17",
    "--use_fast_math",
    "-Xcompiler",
    "-fPIC",
    "-Xptxas",
    "-v",
]


def _nvcc() -> str:
    cand = os.environ.get("NVCC") or shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not Path(cand).exists():
        raise RuntimeError("nvcc not found; set NVCC or install the CUDA toolkit")
    return cand


def _sources(serving: bool = False) -> list[Path]:
    every = sorted(list(CSRC.glob("*.cu")) + list(CSRC.glob("*.cpp")))
    return [p for p in every if p.stem in SERVING_SOURCES] if serving else every


def _flags(src: Path) -> list[str]:
    if src.suffix != ".cu":
        return ["-O3", "-std=c++17", "-Xcompiler", "-fPIC"]
    return [f for f in NVCC_FLAGS if f != "--use_fast_math" or src.stem not in ACCURATE_SOURCES]


def _digest(paths: list[Path]) -> str:
    h = hashlib.sha256()
    for p in sorted(paths + sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h"))):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    for p in sorted(paths):
        h.update(" ".join(_flags(p)).encode())
    return h.hexdigest()


def lib_path(serving: bool = False) -> Path:
    return LIBDIR / (SERVING_LIBNAME if serving else LIBNAME)


def _stamp(serving: bool) -> Path:
    return LIBDIR / ("serving.stamp" if serving else "build.stamp")


def is_current(serving: bool = False) -> bool:
    stamp = _stamp(serving)
    return lib_path(serving).exists() and stamp.exists() and stamp.read_text().strip() == _digest(_sources(serving))


def build(force: bool = False, verbose: bool = False, serving: bool = False) -> Path:
    """Compile every ``csrc/*.cu`` (``serving``: the serving subset) and link the shared object.  Returns its path."""
    srcs = _sources(serving)
    if not srcs:
        raise RuntimeError(f"no CUDA sources in {CSRC}")
    if not force and is_current(serving):
        return lib_path(serving)
    LIBDIR.mkdir(parents=True, exist_ok=True)
    nvcc = _nvcc()
    objs: list[Path] = []
    logs: dict[str, str] = {}

    def compile_one(src: Path) -> Path:
        obj = LIBDIR / (src.stem + ".o")
        cmd = [nvcc, *_flags(src), "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        logs[src.name] = r.stderr + r.stdout
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stderr}\n{r.stdout}")
        return obj

    with ThreadPoolExecutor(max_workers=min(8, len(srcs))) as ex:
        objs = list(ex.map(compile_one, srcs))
    out = lib_path(serving)
    part = out.with_suffix(f".{os.getpid()}.part")  # linked beside its final name: another process never loads half a library
    cmd = [nvcc, "-shared", "-o", str(part), *[str(o) for o in objs], "-gencode", "arch=compute_100a,code=sm_100a", "-ldl", "-lpthread"]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"link failed:\n{r.stderr}")
    os.replace(part, out)
    (LIBDIR / ("ptxas_serving.log" if serving else "ptxas.log")).write_text("\n".join(f"==== {k}\n{v}" for k, v in sorted(logs.items())))
    _stamp(serving).write_text(_digest(srcs))
    if verbose:
        print("\n".join(logs[k] for k in sorted(logs)))
    return out


if __name__ == "__main__":
    p = build(force="--force" in sys.argv, verbose="-v" in sys.argv)
    print(p)
