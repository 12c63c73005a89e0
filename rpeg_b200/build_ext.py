"""In-tree build of the native kernels: ``rpeg_b200/librpeg_kernels.so`` (sm_100a only).

Each ``csrc/*.cu`` is compiled by nvcc (cross-compiles without a GPU) into an object next to the
source and the objects are linked into one shared library that ``rpeg_b200.ops._lib`` loads with
ctypes. Objects are rebuilt only when their source or a header is newer.

``ensure(names)`` is the on-demand form used when a model is loaded: the full library if it is there and up to date,
otherwise a library of just the named sources (the kernels one model family launches), compiled on first use.

Run ``python -m rpeg_b200.build_ext`` (add ``--verbose`` for ptxas register/spill output).
"""
from __future__ import annotations

import concurrent.futures as cf
import fcntl
import os
import shutil
import subprocess
import sys
from pathlib import Path
from typing import Optional, Sequence

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
LIB = PKG / "librpeg_kernels.so"
PART_LIB = PKG / "librpeg_part.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "--use_fast_math",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found (set NVCC or put it on PATH)")


def sources() -> list[Path]:
    return sorted(CSRC.glob("*.cu"))


def _stale(obj: Path, src: Path, headers: list[Path]) -> bool:
    if not obj.exists():
        return True
    t = obj.stat().st_mtime
    return any(p.stat().st_mtime > t for p in [src, *headers])


def _compile(src: Path, verbose: bool) -> tuple[Path, str]:
    obj = src.with_suffix(".o")
    cmd = [_nvcc(), *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
    if verbose:
        cmd[1:1] = ["-Xptxas", "-v"]
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src.name}:\n{res.stdout}\n{res.stderr}")
    return obj, res.stderr


def _headers() -> list[Path]:
    return sorted(CSRC.glob("*.h")) + sorted(CSRC.glob("*.cuh"))


def _build(srcs: list[Path], out: Path, verbose: bool, force: bool) -> Path:
    headers = _headers()
    todo = [s for s in srcs if force or _stale(s.with_suffix(".o"), s, headers)]
    logs: list[str] = []
    if todo:
        with cf.ThreadPoolExecutor(max_workers=min(len(todo), os.cpu_count() or 4)) as ex:
            for obj, log in ex.map(lambda s: _compile(s, verbose), todo):
                logs.append(f"== {obj.name}\n{log}")
    objs = [s.with_suffix(".o") for s in srcs]
    if todo or not out.exists() or any(o.stat().st_mtime > out.stat().st_mtime for o in objs):
        tmp = out.with_suffix(f".{os.getpid()}.tmp.so")
        res = subprocess.run([_nvcc(), "-shared", "-o", str(tmp), *map(str, objs), "-lcudart"], capture_output=True, text=True)
        if res.returncode != 0:
            raise RuntimeError(f"link failed:\n{res.stdout}\n{res.stderr}")
        os.replace(tmp, out)
    if verbose:
        print("\n".join(logs))
    return out


def build(verbose: bool = False, force: bool = False) -> Path:
    return _build(sources(), LIB, verbose, force)


def _fresh(lib: Path, srcs: Sequence[Path]) -> bool:
    return lib.exists() and all(p.stat().st_mtime <= lib.stat().st_mtime for p in (*srcs, *_headers()))


def ensure(names: Optional[Sequence[str]] = None) -> Path:
    """A loadable library with the kernels of ``csrc/<names>`` (None: all of them); compiles what is missing."""
    srcs = sources() if names is None else [CSRC / n for n in names]
    if _fresh(LIB, srcs):
        return LIB
    with open(PKG / ".build.lock.tmp", "w") as lock:          # two first calls must not compile into the same objects
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build(srcs, LIB if names is None else PART_LIB, False, False)


if __name__ == "__main__":
    path = build(verbose="--verbose" in sys.argv, force="--force" in sys.argv)
    print(path)
