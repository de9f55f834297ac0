"""Build recipe for the C-ABI CUDA libraries -- nvcc, sm_100a only.

Usage: python kinetics_b200/build.py [--force] [--verbose] [library ...]   (run by path: importing the
package needs a library this script produces)

  libktk.so         csrc/*.cu: the block top-k paged decode path
  libktk_layers.so  csrc/layers/*.cu plus the host parts they share with it: layer mechanisms with free sizes

Each source is compiled to an object under csrc/build/<library>/ (skipped when the object is newer than
the source and every header), then linked next to this file, so the libraries travel with the tree.
"""
from __future__ import annotations

import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
INCLUDE = PKG.parent / "include"
OUT = PKG / "libktk.so"

#: library -> its sources
LIBRARIES = {
    "libktk": lambda: sorted(CSRC.glob("*.cu")),
    "libktk_layers": lambda: sorted((CSRC / "layers").glob("*.cu")) + [CSRC / "ktk_host.cu", CSRC / "ktk_pool.cu"],
}

NVCC_FLAGS = [
    "-O3", "-std=c++17", "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
    "--expt-relaxed-constexpr", "-Xptxas", "-v",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    raise RuntimeError("nvcc not found")


def build(force: bool = False, verbose: bool = False, library: str = "libktk") -> Path:
    """Compile what is out of date of one library and link it; returns its path."""
    sources = LIBRARIES[library]()
    out = PKG / f"{library}.so"
    headers = sorted(CSRC.glob("*.cuh")) + sorted((CSRC / "layers").glob("*.cuh")) + sorted(INCLUDE.glob("*.h"))
    newest_header = max(h.stat().st_mtime for h in headers)
    objdir = CSRC / "build" / library
    objdir.mkdir(parents=True, exist_ok=True)
    nvcc = _nvcc()

    def compile_one(src: Path):
        obj = objdir / (src.stem + ".o")
        if (not force and obj.exists() and obj.stat().st_mtime > src.stat().st_mtime
                and obj.stat().st_mtime > newest_header):
            return obj, None
        cmd = [nvcc, *NVCC_FLAGS, "-I", str(INCLUDE), "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed on {src.name}:\n{r.stdout}\n{r.stderr}")
        return obj, f"{src.name}\n{r.stderr}"

    with ThreadPoolExecutor(max_workers=min(8, len(sources))) as ex:
        results = list(ex.map(compile_one, sources))
    objs = [o for o, _ in results]
    if verbose:
        for _, log in results:
            if log:
                print(log)
    rebuilt = any(log is not None for _, log in results)
    if rebuilt or force or not out.exists() or any(o.stat().st_mtime > out.stat().st_mtime for o in objs):
        # linked beside its place and moved there, so that a process loading the library never sees half of it
        part = out.with_suffix(f".{os.getpid()}.part")
        cmd = [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", str(part), *map(str, objs)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
        os.replace(part, out)
    return out


def build_all(force: bool = False, verbose: bool = False):
    return [build(force, verbose, name) for name in LIBRARIES]


if __name__ == "__main__":
    names = [a for a in sys.argv[1:] if not a.startswith("-")] or list(LIBRARIES)
    for name in names:
        print(build("--force" in sys.argv, "--verbose" in sys.argv or "-v" in sys.argv, name))
