"""Builds libytensor_cuda.so (sm_100a only) from ytensor_b200/csrc with nvcc.

The library is built in-tree, next to this file, and statically links the CUDA runtime so
that it has no dependency beyond the driver. `python -m ytensor_b200.build` rebuilds what
is out of date; `build(force=True)` rebuilds everything. `build(only=[...])` compiles and links
no more than the named sources (what one model needs: registry.Model.sources) unless a library
that holds them is already there and up to date.
"""
from __future__ import annotations

import fcntl
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG_DIR = Path(__file__).resolve().parent
REPO_DIR = PKG_DIR.parent
CSRC = PKG_DIR / "csrc"
OBJ_DIR = PKG_DIR / "build"
LIB_PATH = PKG_DIR / "libytensor_cuda.so"

NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
    "-I", str(REPO_DIR / "include"),
    *os.environ.get("YTK_NVCC_EXTRA", "").split(),
]


def _sources():
    return sorted(CSRC.glob("*.cu"))


def _newest_header_mtime() -> float:
    hdrs = list(CSRC.glob("*.cuh")) + list((REPO_DIR / "include").glob("*.h"))
    return max((h.stat().st_mtime for h in hdrs), default=0.0)


def _compile(src: Path, verbose: bool) -> Path:
    obj = OBJ_DIR / (src.stem + ".o")
    cmd = [NVCC, *NVCC_FLAGS, "-c", str(src), "-o", str(obj)]
    if verbose:
        cmd.insert(1, "-Xptxas")
        cmd.insert(2, "-v")
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stdout}\n{r.stderr}")
    if verbose:
        sys.stderr.write(r.stderr)
    return obj


def _linked() -> set:
    """Sources (stems) of the library that is there."""
    try:
        return set((OBJ_DIR / "linked.txt").read_text().split()) if LIB_PATH.exists() else set()
    except OSError:
        return set()


def ensure(sources) -> Path:
    """The library with at least the given sources (stems): the one that is there, or one built now. A library shipped
    without its object files is taken as it is when it is newer than every source."""
    sources = set(sources)
    if LIB_PATH.exists():
        newest = max([_newest_header_mtime()] + [(CSRC / (n + ".cu")).stat().st_mtime for n in sources])
        linked = _linked() or {p.stem for p in _sources()}
        if sources <= linked and LIB_PATH.stat().st_mtime >= newest:
            return LIB_PATH
        sources |= _linked()
    return build(only=sources)


def build(force: bool = False, verbose: bool = False, only=None) -> Path:
    OBJ_DIR.mkdir(exist_ok=True)
    with open(OBJ_DIR / ".lock", "w") as lock:  # one build at a time
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build(force, verbose, only)


def _build(force: bool, verbose: bool, only) -> Path:
    hdr_m = _newest_header_mtime()
    todo, objs = [], []
    wanted = [s for s in _sources() if only is None or s.stem in only]
    for src in wanted:
        obj = OBJ_DIR / (src.stem + ".o")
        objs.append(obj)
        if force or not obj.exists() or obj.stat().st_mtime < max(src.stat().st_mtime, hdr_m):
            todo.append(src)
    if todo:
        with ThreadPoolExecutor(max_workers=min(8, len(todo))) as ex:
            list(ex.map(lambda s: _compile(s, verbose), todo))
    names = {s.stem for s in wanted}
    if todo or not LIB_PATH.exists() or _linked() != names:
        cmd = [NVCC, "-shared", "-o", str(LIB_PATH), *map(str, objs), "-cudart", "static",
               "-gencode", "arch=compute_100a,code=sm_100a"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
        (OBJ_DIR / "linked.txt").write_text("\n".join(sorted(names)) + "\n")
    return LIB_PATH


if __name__ == "__main__":
    p = build(force="--force" in sys.argv, verbose="-v" in sys.argv)
    print(p)
