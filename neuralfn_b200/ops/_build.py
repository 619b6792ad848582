"""In-tree build of the sm_100a kernel library and the native runtime pieces.

``build_kernels()`` compiles every ``.cu`` under ``csrc/kernels`` with
``nvcc -gencode arch=compute_100a,code=sm_100a -lineinfo`` into
``neuralfn_b200/lib/libnfn_b200_kernels.so``. nvcc cross-compiles without a GPU,
so the build runs on CPU-only machines; the resulting ``.so`` is what the GPU
machine loads. Objects are rebuilt only when their source (or a header) changed.
"""
from __future__ import annotations

import concurrent.futures
import hashlib
import os
import shutil
import subprocess
import sys
from pathlib import Path

PKG = Path(__file__).resolve().parent.parent
KERNEL_SRC = PKG / "csrc" / "kernels"
RUNTIME_SRC = PKG / "csrc" / "runtime"
ENGINE_SRC = PKG / "csrc" / "engine"
LIB_DIR = PKG / "lib"
OBJ_DIR = PKG / "lib" / "obj"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=default",
]


def _extra_flags() -> list[str]:
    """Extra nvcc flags from ``NFN_EXTRA_NVCC_FLAGS`` (for instance ``-DNFN_KERNEL_TIMERS`` to compile
    the per-role cycle counters into the GEMM and attention kernels). They are part of the object
    digests, so changing them rebuilds."""
    return os.environ.get("NFN_EXTRA_NVCC_FLAGS", "").split()


def _nvcc() -> str:
    for cand in (os.environ.get("NFN_NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found; set NFN_NVCC")


def _digest(paths) -> str:
    h = hashlib.sha256()
    for p in sorted(paths):
        h.update(str(p.name).encode())
        h.update(p.read_bytes())
    h.update(" ".join(NVCC_FLAGS + _extra_flags()).encode())
    return h.hexdigest()


def _compile_one(src: Path, obj: Path, extra: list[str], verbose: bool) -> str:
    lang = ["-x", "cu"] if src.suffix == ".cpp" else []
    cmd = [_nvcc(), *NVCC_FLAGS, *_extra_flags(), *extra, *lang, "-I", str(KERNEL_SRC), "-I", str(ENGINE_SRC), "-c", str(src), "-o", str(obj)]
    proc = subprocess.run(cmd, capture_output=True, text=True)
    if proc.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src.name}:\n{proc.stdout}\n{proc.stderr}")
    return proc.stderr if verbose else ""


# Components: the sources one kind of model needs, built into a library of their own by ``ensure_component``. "all" is the whole library.
COMPONENTS: dict[str, tuple[str, ...]] = {
    "layered": ("common.cu", "gemm_tcgen05.cu", "gemm_2cta.cu", "gemv_bf16.cu", "gemm_skinny.cu", "sampling.cu", "paged_rows.cu", "paged_decode.cu",
                "paged_prefill.cu", "stream_rows.cu", "delta_rows.cu", "delta_chunk.cu", "moe.cu", "moe_rows.cu", "gemm_tp.cu", "head_rows.cu", "latent_decode.cu", "wkv_rows.cu", "wkv_chunk.cu", "linear_rows.cu", "linear_chunk.cu",
                "gru_rows.cu", "engine_core.cpp", "layered_engine.cpp"),
}


def _sources(component: str = "all") -> list[Path]:
    # the resident inference engines (host C++ driving the kernels) live in the same library,
    # so they share the library's CUDA runtime instance and need no extra link step
    every = sorted(KERNEL_SRC.glob("*.cu")) + sorted(ENGINE_SRC.glob("*.cpp"))
    if component == "all":
        return every
    wanted = set(COMPONENTS[component])
    return [s for s in every if s.name in wanted]


def _library(component: str) -> Path:
    return LIB_DIR / ("libnfn_b200_kernels.so" if component == "all" else f"libnfn_b200_{component}.so")


def _object_plan(sources: list[Path]) -> list[tuple[Path, Path, Path, str, bool]]:
    """(source, object, stamp, digest, up to date) per source."""
    headers = sorted(list(KERNEL_SRC.glob("*.h")) + list(KERNEL_SRC.glob("*.cuh")) + list(KERNEL_SRC.glob("*.inc")) +
                     list(ENGINE_SRC.glob("*.h")))
    hdr_digest = _digest(headers)
    plan = []
    for src in sources:
        obj, stamp = OBJ_DIR / (src.stem + ".o"), OBJ_DIR / (src.stem + ".sha")
        want = hashlib.sha256((hdr_digest + _digest([src])).encode()).hexdigest()
        plan.append((src, obj, stamp, want, obj.exists() and stamp.exists() and stamp.read_text() == want))
    return plan


def ensure_component(component: str) -> Path:
    """The library a model of this component runs on: the whole kernel library when it is there and up to date, else the component's
    own, built (or brought up to date) first. One build at a time; others wait for it."""
    import fcntl
    whole = _library("all")
    if whole.exists() and all(p[4] for p in _object_plan(_sources("all"))):
        return whole
    if component == "all":
        return build_kernels()
    OBJ_DIR.mkdir(parents=True, exist_ok=True)
    with open(OBJ_DIR / ".lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return build_kernels(component=component)


def build_kernels(force: bool = False, verbose: bool = False, ptxas_info: bool = False, component: str = "all") -> Path:
    """Compile the CUDA kernel library (or one component of it); returns the path of the shared object."""
    LIB_DIR.mkdir(parents=True, exist_ok=True)
    OBJ_DIR.mkdir(parents=True, exist_ok=True)
    out = _library(component)
    extra = ["-Xptxas", "-v"] if ptxas_info else []
    plan = _object_plan(_sources(component))
    objs = [p[1] for p in plan]
    jobs = [p[:4] for p in plan if force or not p[4]]
    if jobs:
        with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            futs = {ex.submit(_compile_one, s, o, extra, ptxas_info): (s, st, w) for s, o, st, w in jobs}
            for fut in concurrent.futures.as_completed(futs):
                s, st, w = futs[fut]
                log = fut.result()
                st.write_text(w)
                if verbose:
                    print(f"[build] {s.name}", file=sys.stderr)
                if ptxas_info and log:
                    print(log, file=sys.stderr)
    if jobs or not out.exists() or any(o.stat().st_mtime > out.stat().st_mtime for o in objs):
        part = out.with_suffix(f".{os.getpid()}.part")
        cmd = [_nvcc(), "-shared", "-o", str(part), *map(str, objs),
               "-gencode", "arch=compute_100a,code=sm_100a", "-Xcompiler", "-fPIC"]
        proc = subprocess.run(cmd, capture_output=True, text=True)
        if proc.returncode != 0:
            raise RuntimeError(f"link failed:\n{proc.stdout}\n{proc.stderr}")
        os.replace(part, out)
    return out


def build_runtime(force: bool = False, verbose: bool = False) -> list[Path]:
    """Compile the host-side native runtime (C++): one shared object per file
    group under ``csrc/runtime`` (token shards, checkpoint writers, resident
    inference engine). Pure g++, no CUDA needed."""
    LIB_DIR.mkdir(parents=True, exist_ok=True)
    outs = []
    if not RUNTIME_SRC.exists():
        return outs
    sources = sorted(RUNTIME_SRC.glob("*.cpp"))
    if not sources:
        return outs
    headers = sorted(RUNTIME_SRC.glob("*.h"))
    out = LIB_DIR / "libnfn_b200_runtime.so"
    stamp = OBJ_DIR / "runtime.sha"
    OBJ_DIR.mkdir(parents=True, exist_ok=True)
    want = _digest(sources + headers)
    if force or not out.exists() or not stamp.exists() or stamp.read_text() != want:
        cmd = ["g++", "-O2", "-std=c++17", "-fPIC", "-shared", "-Wall", "-Wextra", "-pthread",
               "-I", str(RUNTIME_SRC), "-I", str(KERNEL_SRC), "-o", str(out), *map(str, sources), "-ldl"]
        proc = subprocess.run(cmd, capture_output=True, text=True)
        if proc.returncode != 0:
            raise RuntimeError(f"g++ failed:\n{proc.stdout}\n{proc.stderr}")
        stamp.write_text(want)
        if verbose:
            print("[build] runtime", file=sys.stderr)
    outs.append(out)
    return outs


def build_all(force: bool = False, verbose: bool = False) -> None:
    build_kernels(force=force, verbose=verbose)
    build_runtime(force=force, verbose=verbose)


if __name__ == "__main__":
    build_all(force="--force" in sys.argv, verbose=True)
    if "--ptxas" in sys.argv:
        build_kernels(force=True, verbose=True, ptxas_info=True)
