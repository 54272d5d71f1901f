"""In-tree build of liblumen_b200.so with nvcc for sm_100a.

The shared library links only against the CUDA runtime (NCCL is bound with dlopen at run time),
so it can be loaded from C, C++, Rust or Python.  Objects and the library are written under
``lumen_b200/lib`` and are not tracked by git.  What is out of date is decided by content (a digest of the
source, the headers and the flags beside every object), so a copied or freshly checked out tree is not rebuilt
because of its file times.
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
LIB_DIR = PKG / "lib"
LIB = LIB_DIR / "liblumen_b200.so"
INCLUDE = PKG.parent / "include"

NVCC_FLAGS = [
    "-std=c++17", "-O3", "-lineinfo",
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-Xcompiler", "-fPIC",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found; lumen_b200 has no CPU fallback and cannot be built without CUDA")


def sources() -> list[Path]:
    return sorted(CSRC.glob("*.cu"))


def _digest(paths, extra: str = "") -> str:
    h = hashlib.sha256(extra.encode())
    for p in paths:
        h.update(p.name.encode() + b"\0" + p.read_bytes())
    return h.hexdigest()


def _stale(target: Path, digest: str) -> bool:
    stamp = target.with_suffix(target.suffix + ".sha")
    return not (target.exists() and stamp.exists() and stamp.read_text() == digest)


def _stamp(target: Path, digest: str) -> None:
    target.with_suffix(target.suffix + ".sha").write_text(digest)


def _plan():
    """[(source, object, digest)] and the digest of the library."""
    headers = sorted(CSRC.glob("*.cuh")) + sorted(INCLUDE.glob("*.h"))
    common = _digest(headers, " ".join(NVCC_FLAGS))
    units = [(s, LIB_DIR / (s.stem + ".o"), _digest([s], common)) for s in sources()]
    return units, hashlib.sha256("".join(d for _, _, d in units).encode()).hexdigest()


def up_to_date() -> bool:
    """The library exists and belongs to the sources as they are (needs no compiler)."""
    return not _stale(LIB, _plan()[1])


def build(force: bool = False, verbose: bool = False) -> Path:
    """Compile every .cu under csrc/ and link the shared library.  Returns its path."""
    nvcc = _nvcc()
    LIB_DIR.mkdir(exist_ok=True)
    units, lib_digest = _plan()

    def compile_one(unit):
        src, obj, digest = unit
        if not force and not _stale(obj, digest):
            return None
        cmd = [nvcc, *NVCC_FLAGS, "-Xptxas", "-v", "-c", str(src), "-o", str(obj)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        (LIB_DIR / (src.stem + ".ptxas.log")).write_text(r.stderr)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stderr[-4000:]}")
        _stamp(obj, digest)
        return src.name

    with ThreadPoolExecutor(max_workers=max(1, min(16, len(units), os.cpu_count() or 1))) as ex:
        built = [b for b in ex.map(compile_one, units) if b]
    if built or _stale(LIB, lib_digest):
        cmd = [nvcc, "-shared", "-o", str(LIB), *(str(obj) for _, obj, _ in units), "-ldl"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stderr[-4000:]}")
        _stamp(LIB, lib_digest)
    if verbose:
        print(f"built {built or 'nothing'} -> {LIB}", file=sys.stderr)
    return LIB


if __name__ == "__main__":
    build(force="--force" in sys.argv, verbose=True)
