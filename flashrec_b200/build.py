"""Build the C-ABI shared library ``libflashrec_b200.so`` in-tree with nvcc.

Run as ``python -m flashrec_b200.build`` (or through ``__graft_entry__.build()``).
Every ``csrc/*.cu`` file is compiled for sm_100a only and linked into one shared
object next to this file; objects are rebuilt when a source or header is newer.
"""

from __future__ import annotations

import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path
from typing import Optional, Sequence

HERE = Path(__file__).resolve().parent
CSRC = HERE / "csrc"
OBJ = HERE / "csrc" / "_obj"
LIB = HERE / "libflashrec_b200.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]


def _nvcc() -> str:
    cand = os.environ.get("NVCC") or shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not Path(cand).exists():
        raise RuntimeError("nvcc not found; set NVCC")
    return cand


def _newest_header() -> float:
    hs = list(CSRC.glob("*.cuh")) + list((HERE.parent / "include").glob("*.h"))
    return max(h.stat().st_mtime for h in hs)


def is_current(lib: Path = LIB) -> bool:
    """The library exists and no source or header is newer."""
    srcs = list(CSRC.glob("*.cu"))
    return lib.exists() and lib.stat().st_mtime >= max([_newest_header()] + [s.stat().st_mtime for s in srcs])


def build_subset(name: str, stems: Sequence[str], verbose: bool = False) -> Path:
    """``libflashrec_b200-<name>.so`` from some of the sources only (the entry points one model family calls), or
    the complete library when it is up to date already."""
    if is_current():
        return LIB
    return build(verbose=verbose, stems=stems, lib=HERE / f"libflashrec_b200-{name}.so")


def build(verbose: bool = False, force: bool = False, stems: Optional[Sequence[str]] = None, lib: Path = LIB) -> Path:
    nvcc = _nvcc()
    OBJ.mkdir(exist_ok=True)
    srcs = sorted(CSRC.glob("*.cu")) if stems is None else [CSRC / f"{s}.cu" for s in stems]
    hdr_m = _newest_header()
    jobs = []
    for s in srcs:
        o = OBJ / (s.stem + ".o")
        if force or not o.exists() or o.stat().st_mtime < max(s.stat().st_mtime, hdr_m):
            jobs.append((s, o))

    def compile_one(job):
        s, o = job
        cmd = [nvcc, *NVCC_FLAGS, "-c", str(s), "-o", str(o)]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        r = subprocess.run(cmd, capture_output=True, text=True)
        return s, r

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        for s, r in ex.map(compile_one, jobs):
            if verbose or r.returncode != 0:
                sys.stderr.write(r.stdout + r.stderr)
            if r.returncode != 0:
                raise RuntimeError(f"nvcc failed on {s.name}")
    objs = [str(OBJ / (s.stem + ".o")) for s in srcs]
    if jobs or not lib.exists() or lib.stat().st_mtime < max(Path(o).stat().st_mtime for o in objs):
        cmd = [nvcc, "-shared", "-o", str(lib), *objs, "-gencode", "arch=compute_100a,code=sm_100a"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
    return lib


if __name__ == "__main__":
    print(build(verbose="-v" in sys.argv, force="-f" in sys.argv))
