"""Builds libb200attn.so (sm_100a only) from csrc/*.cu with nvcc, in-tree, next to this file.

    python build.py            # incremental: recompiles sources newer than their object
    python build.py --force
    python build.py --verbose  # adds -Xptxas -v (registers / spills / shared memory per kernel)
    python build.py --part hybrid   # only what that model family needs, as libb200hybrid.so

nvcc cross-compiles, so this runs on a machine without a GPU.
"""
from __future__ import annotations

import argparse
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

HERE = Path(__file__).resolve().parent
CSRC = HERE / "csrc"
INCLUDE = HERE.parent / "include"
OBJ = HERE / "build"
LIB = HERE / "libb200attn.so"

# Sources one model family needs, linked into a library of their own (b200attn/_lib.py loads it when the whole library
# has not been built): what a first run on a machine without built files compiles.
PARTS = {
    "hybrid": (HERE / "libb200hybrid.so", ["paged_kv", "tensor_maps", "layer_glue", "skinny_gemm", "streams", "linear_rnn", "linear_rnn_chunk", "ssd",
                                           "latent", "latent_decode", "latent_prefill_umma", "row_attention", "window", "window_pair_umma"]),
}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    f"-I{INCLUDE}", f"-I{CSRC}",
]


def _nvcc() -> str:
    cand = os.environ.get("NVCC") or "/usr/local/cuda/bin/nvcc"
    return cand if Path(cand).exists() else "nvcc"


def _newest_header() -> float:
    headers = list(CSRC.glob("*.cuh")) + list(CSRC.glob("*.h")) + list(INCLUDE.glob("*.h"))
    return max(h.stat().st_mtime for h in headers)


def ensure(part: str) -> Path:
    """The library a process that only needs `part` loads: the whole one when it is built and newer than the part's
    sources, else the part's own, (re)built if necessary."""
    lib, names = PARTS[part]
    newest = max([_newest_header()] + [(CSRC / f"{n}.cu").stat().st_mtime for n in names])
    if LIB.exists() and LIB.stat().st_mtime >= newest:
        return LIB
    return build(part=part)


def build(force: bool = False, verbose: bool = False, part: str | None = None) -> Path:
    out = LIB
    if part is None:
        sources = sorted(CSRC.glob("*.cu"))
    else:
        out, names = PARTS[part]
        sources = [CSRC / f"{n}.cu" for n in names]
    if not sources:
        raise RuntimeError(f"no CUDA sources under {CSRC}")
    OBJ.mkdir(exist_ok=True)
    hdr_time = _newest_header()
    jobs = []
    for src in sources:
        obj = OBJ / (src.stem + ".o")
        stale = force or not obj.exists() or obj.stat().st_mtime < max(src.stat().st_mtime, hdr_time)
        if stale:
            cmd = [_nvcc(), *NVCC_FLAGS, *(["-Xptxas", "-v"] if verbose else []), "-c", str(src), "-o", str(obj)]
            jobs.append((src, cmd))

    def run(job):
        src, cmd = job
        res = subprocess.run(cmd, capture_output=True, text=True)
        return src, res

    failed = False
    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as pool:
        for src, res in pool.map(run, jobs):
            if verbose or res.returncode != 0:
                sys.stderr.write(f"--- {src.name}\n{res.stdout}{res.stderr}\n")
            failed |= res.returncode != 0
    if failed:
        raise RuntimeError("nvcc failed (see stderr)")
    objs = [str(OBJ / (s.stem + ".o")) for s in sources]
    if jobs or not out.exists() or out.stat().st_mtime < max(Path(o).stat().st_mtime for o in objs):
        link = [_nvcc(), "-shared", "-o", str(out), *objs, "-gencode", "arch=compute_100a,code=sm_100a",
                "-Xcompiler", "-fPIC", "-lcudart"]
        res = subprocess.run(link, capture_output=True, text=True)
        if res.returncode != 0:
            sys.stderr.write(res.stdout + res.stderr)
            raise RuntimeError("link failed")
    return out


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    ap.add_argument("--part", choices=sorted(PARTS))
    a = ap.parse_args()
    print(build(force=a.force, verbose=a.verbose, part=a.part))
