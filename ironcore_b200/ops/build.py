"""Build the native sm_100a library in-tree with nvcc.

Every ``csrc/*.cu`` file is compiled with
``-gencode arch=compute_100a,code=sm_100a -lineinfo`` into an object file and the
objects are linked into ``ironcore_b200/ops/_native/libironcore_b200.so``. nvcc
cross-compiles without a GPU, so the build runs on a CPU-only machine; the
resulting ``.so`` is loaded through :mod:`ctypes` (plain C ABI, no torch headers,
seconds per file).

A checkout that was never built compiles on first use, and then only what is used: every source file is a
unit of its own (``build_unit``), a shared library named after its sources' digest that exports the entry points
found in that file. :mod:`.native` looks symbols up in the complete library when it is current and in the units
otherwise.

Usage: ``python -m ironcore_b200.ops.build [--force] [--verbose]``
"""

from __future__ import annotations

import hashlib
import json
import os
import re
import shutil
import subprocess
import sys
import tempfile
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

REPO_ROOT = Path(__file__).resolve().parents[2]
CSRC = REPO_ROOT / "csrc"
OUT_DIR = Path(__file__).resolve().parent / "_native"
LIB_PATH = OUT_DIR / "libironcore_b200.so"
STAMP = OUT_DIR / "build_stamp.json"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "-Xcompiler", "-fvisibility=hidden",
    "-diag-suppress", "177",
]


def _nvcc() -> str:
    cand = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(cand):
        raise RuntimeError("nvcc not found; cannot build the sm_100a kernels")
    return cand


def _sources():
    return sorted(CSRC.glob("*.cu"))


def _digest() -> str:
    h = hashlib.sha256()
    for p in sorted(list(CSRC.glob("*.cu")) + list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h"))):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    h.update(" ".join(NVCC_FLAGS).encode())
    return h.hexdigest()


def is_current() -> bool:
    if not LIB_PATH.exists() or not STAMP.exists():
        return False
    try:
        return json.loads(STAMP.read_text()).get("digest") == _digest()
    except Exception:
        return False


def build(force: bool = False, verbose: bool = False) -> Path:
    """Compile all kernels (if sources changed) and return the library path."""
    if not force and is_current():
        return LIB_PATH
    OUT_DIR.mkdir(parents=True, exist_ok=True)
    nvcc = _nvcc()
    objs = []

    def compile_one(src: Path):
        obj = OUT_DIR / (src.stem + ".o")
        cmd = [nvcc, *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            sys.stderr.write(r.stderr)
        return obj

    with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 2)) as ex:
        objs = list(ex.map(compile_one, _sources()))
    link = [nvcc, "-shared", "-o", str(LIB_PATH), *map(str, objs),
            "-gencode", "arch=compute_100a,code=sm_100a", "-Xcompiler", "-fPIC"]
    r = subprocess.run(link, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    STAMP.write_text(json.dumps({"digest": _digest(), "sources": [s.name for s in _sources()]}))
    return LIB_PATH


# --------------------------------------------------------------------------- units
# host functions that one source file takes from another
_UNIT_PARTNERS = {"flash_bwd": ("flash_fwd",)}
_EXPORT = re.compile(r"^ICB_API\s+int\s+(icb_\w+)\s*\(", re.M)


def exported_symbols() -> dict:
    """Entry point name -> stem of the ``csrc/*.cu`` file that defines it."""
    return {name: src.stem for src in _sources() for name in _EXPORT.findall(src.read_text())}


def unit_path(stem: str) -> Path:
    """Where the library of one source file lives; the name changes with the sources, the headers and the flags."""
    h = hashlib.sha256()
    files = [CSRC / f"{s}.cu" for s in (stem, *_UNIT_PARTNERS.get(stem, ()))]
    for p in files + sorted(list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h"))):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    h.update(" ".join(NVCC_FLAGS).encode())
    return OUT_DIR / f"libicb_{stem}_{h.hexdigest()[:16]}.so"


def build_unit(stem: str) -> Path:
    """Compile one source file (and its partners) into its own shared library unless that exists already."""
    path = unit_path(stem)
    if path.exists():
        return path
    OUT_DIR.mkdir(parents=True, exist_ok=True)
    sources = [str(CSRC / f"{s}.cu") for s in (stem, *_UNIT_PARTNERS.get(stem, ()))]
    fd, part = tempfile.mkstemp(dir=OUT_DIR, prefix=f".{stem}_", suffix=".so")     # another process may build it too
    os.close(fd)
    try:
        r = subprocess.run([_nvcc(), *NVCC_FLAGS, "-I", str(CSRC), "-shared", "-o", part, *sources],
                           capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {stem}.cu:\n{r.stdout}\n{r.stderr}")
        os.chmod(part, 0o755)
        os.replace(part, path)
    finally:
        if os.path.exists(part):
            os.unlink(part)
    return path


def build_units(stems) -> None:
    stems = sorted(set(stems))
    with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 2)) as ex:
        list(ex.map(build_unit, stems))


if __name__ == "__main__":
    path = build(force="--force" in sys.argv, verbose="--verbose" in sys.argv)
    print(path)
