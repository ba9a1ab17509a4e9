"""Builds the in-tree CUDA libraries for sm_100a with plain ``nvcc``.

The kernels expose a C ABI (raw pointers + ``cudaStream_t``) and are loaded with ``ctypes``, so the
libraries have no dependency on PyTorch headers, compile in seconds and cross-compile on a machine
without a GPU.  ``python -m mfq_b200.ops.build`` rebuilds them; ``build(force=False)`` is incremental.

* ``_mfq_b200_kernels.so`` -- the FP8 / packed / collective kernels and the engine's bookkeeping;
* ``_mfq_b200_dense.so`` -- the unquantized path (:data:`DENSE_SOURCES`), on its own so that a model that only needs it
  can be built in a few seconds (``build(only="dense")``).
"""

from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

HERE = Path(__file__).resolve().parent
CSRC = HERE / "csrc"
LIB_PATH = HERE / "_mfq_b200_kernels.so"
DENSE_LIB_PATH = HERE / "_mfq_b200_dense.so"
DENSE_SOURCES = ("dense_gemm.cu", "dense_moe.cu", "stream_ops.cu", "mix_ops.cu", "window_attn.cu", "window_attn_prefill.cu",
                 "window_attn_prefill_bias.cu", "latent_attn.cu", "gla.cu", "gla_chunk.cu", "delta.cu", "delta_chunk.cu", "ssd.cu", "ssd_chunk.cu", "moe_route.cu")
SHARED_SOURCES = ("moe_route.cu",)  # part of the main library too
OBJ_DIR = HERE / "build"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--expt-relaxed-constexpr", "-Xcompiler", "-fPIC", "-Xptxas", "-v",
]


def nvcc_path() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found: the CUDA kernels cannot be built")


def sources() -> list[Path]:
    return sorted(CSRC.glob("*.cu"))


def _digest(path: Path) -> str:
    h = hashlib.sha256()
    h.update(path.read_bytes())
    for header in sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h")):
        h.update(header.read_bytes())
    h.update(" ".join(NVCC_FLAGS).encode())
    return h.hexdigest()


def _compile_one(src: Path, force: bool) -> tuple[Path, str]:
    obj = OBJ_DIR / (src.stem + ".o")
    stamp = OBJ_DIR / (src.stem + ".sha")
    digest = _digest(src)
    if not force and obj.exists() and stamp.exists() and stamp.read_text() == digest:
        return obj, ""
    cmd = [nvcc_path(), *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
    proc = subprocess.run(cmd, capture_output=True, text=True)
    if proc.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src.name}:\n{proc.stderr}")
    stamp.write_text(digest)
    return obj, proc.stderr


def libraries() -> dict[str, tuple[Path, list[Path]]]:
    """Library name -> (path, its sources)."""
    dense = [p for p in sources() if p.name in DENSE_SOURCES]
    return {"kernels": (LIB_PATH, [p for p in sources() if p not in dense or p.name in SHARED_SOURCES]), "dense": (DENSE_LIB_PATH, dense)}


def _link(path: Path, objs: list[Path]) -> None:
    part = path.with_suffix(f".{os.getpid()}.part")  # a process that loads the library never sees half of it
    proc = subprocess.run([nvcc_path(), "--shared", "-o", str(part), *map(str, objs)], capture_output=True, text=True)
    if proc.returncode != 0:
        raise RuntimeError(f"link failed:\n{proc.stderr}")
    os.replace(part, path)


def build(force: bool = False, verbose: bool = False, only: str | None = None) -> Path:
    """Compile ``csrc/*.cu`` and link the shared libraries (``only``: just the one of that name).  Returns the path of the
    library asked for, by default the main one."""
    OBJ_DIR.mkdir(exist_ok=True)
    libs = libraries()
    chosen = libs if only is None else {only: libs[only]}
    srcs = sorted({s for _, group in chosen.values() for s in group})
    with ThreadPoolExecutor(max_workers=min(8, len(srcs))) as pool:
        results = dict(zip(srcs, pool.map(lambda s: _compile_one(s, force), srcs)))
    log = "".join(text for _, text in results.values())
    if log:
        (OBJ_DIR / "ptxas.log").write_text(log)
    for path, group in chosen.values():
        if not path.exists() or any(results[s][1] or results[s][0].stat().st_mtime > path.stat().st_mtime for s in group):
            _link(path, [results[s][0] for s in group])
    if verbose and log:
        print(log, file=sys.stderr)
    return libs[only or "kernels"][0]


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose=True))
