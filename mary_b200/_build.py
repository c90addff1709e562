"""Builds the native libraries in-tree.

Two shared objects are produced next to this file:

* ``_core.so``    — C++17 host runtime: pile store, BLAKE3, paged-KV allocator, batch scheduler
                   (compiled with g++).
* ``_kernels.so`` — every CUDA kernel, compiled by nvcc for sm_100a only.  The launchers are plain
                   ``extern "C"`` functions taking raw device pointers and a stream, so the library
                   has no dependency on torch headers and builds in seconds per file.

Both are loaded with ctypes (``mary_b200._native``).
"""
from __future__ import annotations

import concurrent.futures as cf
import hashlib
import os
import shutil
import subprocess
import sys
from pathlib import Path

ROOT = Path(__file__).resolve().parent
CSRC = ROOT / "csrc"
OBJ = ROOT / "csrc" / "build"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr", "-Xptxas", "-v",
]
# Files whose arithmetic also serves 32-bit models keep the exact divide, square root and exponential; all others use the fast forms.
EXACT_MATH = {"linear_attention", "recurrent_scan", "residual32", "parallel_stream", "gemm_simt", "attention_general", "latent", "state_space", "ssd_chunk",
              "hyper_streams"}


def _stamp(paths, extra=""):
    h = hashlib.sha256(extra.encode())
    for p in sorted(paths):
        h.update(Path(p).name.encode())
        h.update(Path(p).read_bytes())
    return h.hexdigest()


def _run(cmd, log=None):
    r = subprocess.run(cmd, capture_output=True, text=True)
    if log is not None:
        Path(log).write_text(r.stdout + r.stderr)
    if r.returncode != 0:
        sys.stderr.write(r.stdout + r.stderr)
        raise RuntimeError("build failed: " + " ".join(map(str, cmd)))
    return r.stdout + r.stderr


def build_core(force: bool = False) -> Path:
    out = ROOT / "_core.so"
    srcs = sorted((CSRC / "core").glob("*.cpp"))
    hdrs = sorted((CSRC / "core").glob("*.hpp"))
    stamp = _stamp(srcs + hdrs)
    sf = OBJ / "core.stamp"
    if out.exists() and not force and sf.exists() and sf.read_text() == stamp:
        return out
    OBJ.mkdir(parents=True, exist_ok=True)
    cxx = shutil.which("g++") or "g++"
    _run([cxx, "-O3", "-std=c++17", "-fPIC", "-shared", "-pthread", "-o", str(out)] + [str(s) for s in srcs])
    sf.write_text(stamp)
    return out


def nvcc_path() -> str:
    return shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"


def _kernel_sources(only=None):
    """``[(source, compile flags, stamp of everything the object depends on)]`` of all kernels, or of the files named in ``only``."""
    srcs = sorted((CSRC / "kernels").glob("*.cu"))
    if only is not None:
        missing = set(only) - {s.stem for s in srcs}
        if missing:
            raise ValueError(f"no kernel source named {sorted(missing)}")
        srcs = [s for s in srcs if s.stem in only]
    hdrs = sorted((CSRC / "kernels").glob("*.cuh")) + sorted((CSRC / "kernels").glob("*.h"))
    hdr_stamp = _stamp(hdrs, " ".join(NVCC_FLAGS))
    out = []
    for src in srcs:
        flags = NVCC_FLAGS + ([] if src.stem in EXACT_MATH else ["--use_fast_math"])
        out.append((src, flags, _stamp([src], hdr_stamp + " ".join(flags))))
    return out


def build_kernels(force: bool = False, only=None) -> Path:
    """Compile and link every kernel into ``_kernels.so``, or the sources named in ``only`` into ``_kernels_part.so``."""
    out = ROOT / ("_kernels.so" if only is None else "_kernels_part.so")
    OBJ.mkdir(parents=True, exist_ok=True)
    nvcc = nvcc_path()

    def compile_one(item):
        src, flags, stamp = item
        obj = OBJ / (src.stem + ".o")
        sf = OBJ / (src.stem + ".stamp")
        if obj.exists() and not force and sf.exists() and sf.read_text() == stamp:
            return obj, False
        _run([nvcc] + flags + ["-I", str(CSRC / "kernels"), "-c", str(src), "-o", str(obj)],
             log=OBJ / (src.stem + ".ptxas.log"))
        sf.write_text(stamp)
        return obj, True

    items = _kernel_sources(only)
    with cf.ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 2)) as ex:
        res = list(ex.map(compile_one, items))
    objs = [str(o) for o, _ in res]
    linked = OBJ / (out.name + ".stamp")
    stamp = _stamp([], " ".join(s for _, _, s in items))
    if out.exists() and not force and linked.exists() and linked.read_text() == stamp:
        return out
    tmp = out.with_suffix(f".{os.getpid()}.tmp")           # renamed into place: another process never loads a half-written library
    _run([nvcc, "-shared", "-o", str(tmp)] + objs + ["-gencode", "arch=compute_100a,code=sm_100a", "-lcudart"])
    os.replace(tmp, out)
    linked.write_text(stamp)
    return out


def ensure_kernels(only) -> Path:
    """A library that holds at least the sources named in ``only``: the full one when it has been built from the sources as they are,
    else a partial one, compiled now if need be."""
    full, stamp_file = ROOT / "_kernels.so", OBJ / "_kernels.so.stamp"
    if full.exists() and (not stamp_file.exists() or stamp_file.read_text() == _stamp([], " ".join(s for _, _, s in _kernel_sources()))):
        return full
    return build_kernels(only=only)


def build_all(force: bool = False):
    return build_core(force), build_kernels(force)


if __name__ == "__main__":
    print(build_all("--force" in sys.argv))
