"""Builds the sm_100a kernel library in-tree with nvcc.

Every ``*.cu`` file next to this script is compiled to an object file under
``csrc/build/`` and the objects are linked into ``easydel_b200/lib/libedl_b200.so``.
The library has a plain C ABI (``extern "C"`` launchers taking raw device pointers
and a stream handle) and is loaded with ``ctypes``; no Python headers are needed,
so a file compiles in seconds and cross-compiles on a machine without a GPU.

Run ``python -m easydel_b200.csrc.build`` (add ``--force`` to rebuild everything,
``--verbose`` for ptxas register/shared-memory reports). ``EDL_NVCC_EXTRA`` adds compiler flags, and
``--out PATH`` links the result somewhere else, so that a checking build
(``EDL_NVCC_EXTRA=-DEDL_BOUNDS_CHECK python -m easydel_b200.csrc.build --out /tmp/libedl_check.so``, loaded
with ``EDL_LIB_PATH``) can sit beside the production library.
"""

from __future__ import annotations

import argparse
import concurrent.futures as cf
import hashlib
import json
import os
import shutil
import subprocess
import sys
from pathlib import Path

CSRC = Path(__file__).resolve().parent
PKG = CSRC.parent
BUILD = CSRC / "build"
LIB_DIR = PKG / "lib"
LIB_PATH = LIB_DIR / "libedl_b200.so"

NVCC_FLAGS = [
    "-gencode",
    "arch=compute_100a,code=sm_100a",
    "-lineinfo",
    "-O3",
    "-std=c++17",
    "--use_fast_math",
    "-Xcompiler",
    "-fPIC",
    "-Xcompiler",
    "-fvisibility=hidden",
    "--expt-relaxed-constexpr",
]

# Kernels whose job is 32-bit arithmetic (fp32 residual stream, gates and recurrences, attention of fp32 models) are
# compiled without fast-math.
PRECISE = frozenset({"stream_ops", "hgrn2", "gdelta", "attention_simt", "latent_ops", "moe_serving"})

# What serving a model family needs, by model type, for a first call on a machine without a built library.
SERVING_PARTS = {
    "rakevik": ("common", "gemm", "attention_fwd", "attention_decode", "attn_combine", "attention_simt", "serving",
                "host_native", "stream_ops", "hgrn2"),
    "disunex": ("common", "gemm", "attention_fwd", "attention_mla_decode", "attn_combine", "attention_simt", "serving",
                "host_native", "stream_ops", "latent_ops", "moe", "moe_serving"),
    "gasetar": ("common", "gemm", "attention_fwd", "attention_decode", "attention_mla_decode", "attn_combine",
                "attention_simt", "serving", "host_native", "stream_ops", "latent_ops", "moe", "moe_serving", "norm_act"),
    "ninisun": ("common", "gemm", "attention_fwd", "attention_decode", "attn_combine", "attention_simt", "serving",
                "host_native", "stream_ops", "gdelta", "norm_act"),
}
MANIFEST_SUFFIX = ".sources.json"      # beside a linked library: the digest of every source it was built from


def _nvcc() -> str:
    cand = os.environ.get("NVCC") or shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not Path(cand).exists():
        raise RuntimeError("nvcc not found; set NVCC or put it on PATH")
    return cand


def _flags_for(src: Path, flags: list[str]) -> list[str]:
    return [f for f in flags if f != "--use_fast_math"] if src.stem in PRECISE else flags


def _digest(src: Path, flags: list[str]) -> str:
    flags = _flags_for(src, flags)
    h = hashlib.sha256()
    h.update(" ".join(flags).encode())
    h.update(src.read_bytes())
    for hdr in sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h")):
        h.update(hdr.read_bytes())
    return h.hexdigest()


def _compile_one(nvcc: str, src: Path, flags: list[str], force: bool, verbose: bool) -> tuple[Path, bool, str]:
    obj = BUILD / (src.stem + ".o")
    stamp = BUILD / (src.stem + ".sha")
    dig = _digest(src, flags)
    if not force and obj.exists() and stamp.exists() and stamp.read_text() == dig:
        return obj, False, ""
    cmd = [nvcc, *_flags_for(src, flags), "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
    proc = subprocess.run(cmd, capture_output=True, text=True)
    if proc.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src.name}:\n{proc.stdout}\n{proc.stderr}")
    stamp.write_text(dig)
    return obj, True, (proc.stderr if verbose else "")


def sources() -> list[Path]:
    return sorted(CSRC.glob("*.cu"))


def _manifest(lib: Path) -> dict[str, str]:
    try:
        return json.loads(lib.with_name(lib.name + MANIFEST_SUFFIX).read_text())
    except (OSError, ValueError):
        return {}


def ensure(model_type: str) -> Path:
    """A library with current kernels for serving ``model_type``: the full one if it is up to date in the parts the
    family needs, else a smaller one with those parts only (compiled and linked now if it is missing or stale)."""
    parts = SERVING_PARTS.get(model_type)
    if parts is None:
        return build()
    want = {n: _digest(CSRC / f"{n}.cu", list(NVCC_FLAGS)) for n in parts}
    partial = LIB_DIR / f"libedl_b200_{model_type}.so"
    for lib in (LIB_PATH, partial):
        have = _manifest(lib)
        if lib.exists() and all(have.get(n) == d for n, d in want.items()):
            return lib
    return build(only=parts, link=partial)


def build(force: bool = False, verbose: bool = False, jobs: int | None = None, out: str | None = None,
          only: tuple[str, ...] | None = None, link: Path | None = None) -> Path:
    """Compiles what changed and links the shared library; returns its path. ``out``: link there instead of the
    in-tree location, with the objects in a directory of their own (a build with other flags beside the main one).
    ``only``: the sources to take, by stem; ``link``: where to link them."""
    global BUILD, LIB_PATH
    nvcc = _nvcc()
    if out is not None:
        LIB_PATH = Path(out).resolve()
        BUILD = CSRC / "build" / ("alt-" + hashlib.sha256(str(LIB_PATH).encode()).hexdigest()[:8])
        BUILD.mkdir(parents=True, exist_ok=True)
        LIB_PATH.parent.mkdir(parents=True, exist_ok=True)
    BUILD.mkdir(exist_ok=True)
    LIB_DIR.mkdir(exist_ok=True)
    flags = list(NVCC_FLAGS)
    extra = os.environ.get("EDL_NVCC_EXTRA", "").split()   # e.g. -DEDL_BOUNDS_CHECK for a checking build
    flags += extra
    if verbose:
        flags += ["-Xptxas", "-v"]
    srcs = sources() if only is None else [CSRC / f"{n}.cu" for n in only]
    target = LIB_PATH if link is None else link
    objs: list[Path] = []
    changed = False
    with cf.ThreadPoolExecutor(max_workers=jobs or min(8, os.cpu_count() or 4)) as ex:
        futs = [ex.submit(_compile_one, nvcc, s, flags, force, verbose) for s in srcs]
        for f in futs:
            obj, did, log = f.result()
            objs.append(obj)
            changed |= did
            if log:
                print(log, file=sys.stderr)
    digests = {x.stem: _digest(x, flags) for x in srcs}
    if changed or not target.exists() or _manifest(target) != digests:
        tmp = target.with_suffix(".so.tmp")
        cmd = [nvcc, "-shared", "-o", str(tmp), *map(str, objs), "-gencode", "arch=compute_100a,code=sm_100a",
               "-lcudart_static", "-Xcompiler", "-fPIC"]
        proc = subprocess.run(cmd, capture_output=True, text=True)
        if proc.returncode != 0:
            raise RuntimeError(f"link failed:\n{proc.stdout}\n{proc.stderr}")
        os.replace(tmp, target)
        target.with_name(target.name + MANIFEST_SUFFIX).write_text(json.dumps(digests))
    return target


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__)
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    ap.add_argument("-j", "--jobs", type=int, default=None)
    ap.add_argument("--out", default=None, help="link the library here instead of easydel_b200/lib/")
    a = ap.parse_args()
    print(build(force=a.force, verbose=a.verbose, jobs=a.jobs, out=a.out))


if __name__ == "__main__":
    main()
