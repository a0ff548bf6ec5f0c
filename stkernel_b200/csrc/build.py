"""Build the CUDA library in-tree: ``python -m stkernel_b200.csrc.build``.

Every ``.cu`` file here is compiled for sm_100a only and linked into
``stkernel_b200/_lib/libstk_b200.so`` (plain ``extern "C"`` entry points, loaded
with ctypes; no torch headers, so a file compiles in seconds and the library has
no ABI tie to a torch build).  Objects are rebuilt only when their source or a
header is newer.

`build(only=[...])` compiles just the named files into a library of its own (`libstk_b200-<name>.so`): what one model family
needs, for a checkout whose first command should not wait for kernels it never launches.
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path
from typing import Optional, Sequence

HERE = Path(__file__).resolve().parent
OUT_DIR = HERE.parent / "_lib"
OBJ_DIR = HERE.parent.parent / "build" / "obj"
LIB = OUT_DIR / "libstk_b200.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden", "--expt-relaxed-constexpr",
]


def sources(only: Optional[Sequence[str]] = None) -> list[Path]:
    if only is None:
        return sorted(HERE.glob("*.cu"))
    return [HERE / n for n in sorted(only)]


def headers() -> list[Path]:
    """What the sources include (the `.h` files are interfaces for other programs, generated or hand-written)."""
    return sorted(HERE.glob("*.cuh"))


def source_digest(only: Optional[Sequence[str]] = None) -> str:
    """Hash of everything the library is made from (file times say nothing in a fresh checkout or a copied tree)."""
    h = hashlib.sha256(" ".join(NVCC_FLAGS).encode())
    for f in sources(only) + headers():
        h.update(f.name.encode() + b"\0" + f.read_bytes())
    return h.hexdigest()


def library_path(name: Optional[str] = None) -> Path:
    return LIB if name is None else OUT_DIR / f"libstk_b200-{name}.so"


def is_current(lib: Path, only: Optional[Sequence[str]] = None) -> bool:
    """Whether `lib` exists and was linked from the sources as they are now."""
    key = lib.with_suffix(".key")
    return lib.exists() and key.exists() and key.read_text().strip() == source_digest(only)


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found (PATH, /usr/local/cuda/bin)")
    return exe


def _newest_header() -> float:
    return max((h.stat().st_mtime for h in headers()), default=0.0)


def _compile(src: Path, verbose: bool) -> Path:
    obj = OBJ_DIR / (src.stem + ".o")
    stamp = max(src.stat().st_mtime, _newest_header())
    if obj.exists() and obj.stat().st_mtime >= stamp:
        return obj
    cmd = [_nvcc(), *NVCC_FLAGS, "-c", str(src), "-o", str(obj)]
    if verbose:
        cmd.insert(1, "-Xptxas")
        cmd.insert(2, "-v")
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stdout}\n{r.stderr}")
    if verbose:
        sys.stderr.write(r.stderr)
    return obj


def build(verbose: bool = False, force: bool = False, only: Optional[Sequence[str]] = None, name: Optional[str] = None) -> Path:
    """Compile what changed and link.  only + name: a library of those files alone."""
    OUT_DIR.mkdir(parents=True, exist_ok=True)
    OBJ_DIR.mkdir(parents=True, exist_ok=True)
    if force:
        for o in OBJ_DIR.glob("*.o"):
            o.unlink()
    lib = library_path(name)
    digest = source_digest(only)
    srcs = sources(only)
    # the longest compilations first
    srcs.sort(key=lambda f: -f.stat().st_size)
    with ThreadPoolExecutor(max_workers=min(16, os.cpu_count() or 1)) as ex:
        objs = list(ex.map(lambda s: _compile(s, verbose), srcs))
    if (not lib.exists()) or any(o.stat().st_mtime > lib.stat().st_mtime for o in objs):
        part = lib.with_suffix(f".{os.getpid()}.part")
        cmd = [_nvcc(), "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", str(part),
               *[str(o) for o in objs], "-lcudart"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
        os.replace(part, lib)                     # a process that has the old file open keeps it
    lib.with_suffix(".key").write_text(digest + "\n")
    return lib


if __name__ == "__main__":
    print(build(verbose="-v" in sys.argv, force="--force" in sys.argv))
