"""Compiles this package's CUDA sources for sm_100a into shared libraries.

Kinds of library: ``core`` (kernels whose sizes are run-time arguments),
``attn_d<D>`` (the attention kernels, compiled once per head size D with
``-DKRK_HEAD_DIM=D``, so a model compiles only the head size it has), ``mix``
(the kernels of models with a 32-bit residual stream, windowed attention with a
sink or over latent rows), ``scan`` (recurrent state), ``memory`` (matrix states
without a removal term) and ``moe`` (routed
experts); each of the last four is compiled and loaded when a model first calls
one of its kernels, so a model compiles what it needs; ``latent_k<D>_v<P>`` (prompt
attention over keys and values made from latent rows, per pair of sizes, likewise). A library
is rebuilt when a source or a flag changes (its name carries a hash of both) and
is otherwise loaded as it is. Libraries live in ``csrc/_build`` inside the
package when that is writable, else under ``$KRK_BUILD_DIR`` or a per-user
folder in the system's temporary directory; no home directory and no network are
needed. While nvcc runs, a line is printed every few seconds.
"""

from __future__ import annotations

import fcntl
import hashlib
import os
import shutil
import subprocess
import sys
import tempfile
import threading
import time
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

SRC_DIR = Path(__file__).parent

CORE_SOURCES = ["elementwise.cu", "rope_kv.cu", "gemm_simple.cu", "select.cu", "skinny_bf16.cu", "gemm_tcgen05.cu", "lt_gemm.cu"]
CORE_LIBS = ["-lcublasLt"]  # lt_gemm.cu; the process already holds the copy that torch loaded
MIX_SOURCES = ["wide_rows.cu", "sink_attention.cu", "latent.cu", "hyper.cu", "mixed_attention.cu", "latent_decode.cu"]
SCAN_SOURCES = ["recurrent.cu", "ssd.cu"]
MEMORY_SOURCES = ["matrix_memory.cu", "matrix_memory_chunks.cu", "matrix_memory_step.cu"]
MOE_SOURCES = ["routed.cu", "grouped_gemm.cu"]
SMALL_LIBRARIES = {"mix": MIX_SOURCES, "scan": SCAN_SOURCES, "memory": MEMORY_SOURCES, "moe": MOE_SOURCES}
LATENT_SOURCES = ["latent_prefill.cu"]
ATTN_SOURCES = ["attention_simple.cu", "attention_mma.cu", "attention_tcgen05.cu"]
HEADERS = ["common.cuh", "mma.cuh", "tcgen05.cuh", "attention_noalloc.h"]

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden"]
# extra flags for performance work, e.g. KRK_EXTRA_NVCC_FLAGS="-DKRK_TRACE"; they are part of the library's hash
NVCC_FLAGS += os.environ.get("KRK_EXTRA_NVCC_FLAGS", "").split()


class BuildError(RuntimeError):
    pass


def _say(msg: str) -> None:
    print(f"[kernel_rush_kawk_b200 build] {msg}", file=sys.stderr, flush=True)


def find_nvcc() -> str:
    for cand in (os.environ.get("KRK_NVCC"), shutil.which("nvcc"),
                 os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "bin", "nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.isfile(cand) and os.access(cand, os.X_OK):
            return cand
    raise BuildError("nvcc was not found (looked at $KRK_NVCC, PATH, $CUDA_HOME/bin, /usr/local/cuda/bin); "
                     "the CUDA extension cannot be compiled and this library has no other compute path")


def build_dir() -> Path:
    cands = []
    if os.environ.get("KRK_BUILD_DIR"):
        cands.append(Path(os.environ["KRK_BUILD_DIR"]))
    cands.append(SRC_DIR / "_build")
    cands.append(Path(tempfile.gettempdir()) / f"kernel_rush_kawk_b200_build_{os.getuid()}")
    for d in cands:
        try:
            d.mkdir(parents=True, exist_ok=True)
            fd, probe = tempfile.mkstemp(prefix=".probe_", dir=d)  # a name of its own: threads and processes probe at once
            os.close(fd)
            os.unlink(probe)
            return d
        except OSError:
            continue
    raise BuildError(f"no writable folder for compiled kernels among {[str(c) for c in cands]}")


def _existing(sources):
    return [s for s in sources if (SRC_DIR / s).is_file()]


def _key(sources, defines, libs=None) -> str:
    h = hashlib.sha256()
    for name in list(sources) + _existing(HEADERS):
        h.update(name.encode())
        h.update((SRC_DIR / name).read_bytes())
    h.update(" ".join(NVCC_FLAGS + list(defines) + (list(libs) if libs is not None else CORE_LIBS)).encode())
    return h.hexdigest()[:12]


def library_path(kind: str, head_dim=None) -> tuple[Path, list, list]:
    """``head_dim``: the head size of an "attn" library, the (key, value) sizes of a "latent" one."""
    if kind == "latent":
        sources, (key, value) = _existing(LATENT_SOURCES), (int(n) for n in head_dim)
        defines = [f"-DKRK_KEY_DIM={key}", f"-DKRK_VALUE_DIM={value}"]
        return build_dir() / f"libkrk_latent_k{key}_v{value}_{_key(sources, defines, [])}.so", sources, defines
    if kind == "core":
        sources, defines, stem = _existing(CORE_SOURCES), [], "libkrk_core"
    elif kind in SMALL_LIBRARIES:
        sources, defines, stem = _existing(SMALL_LIBRARIES[kind]), [], f"libkrk_{kind}"
        return build_dir() / f"{stem}_{_key(sources, defines, [])}.so", sources, defines
    else:
        sources, defines, stem = _existing(ATTN_SOURCES), [f"-DKRK_HEAD_DIM={int(head_dim)}"], f"libkrk_attn_d{int(head_dim)}"
    return build_dir() / f"{stem}_{_key(sources, defines)}.so", sources, defines


def _compile_one(nvcc: str, src: Path, obj: Path, defines) -> None:
    cmd = [nvcc, *NVCC_FLAGS, *defines, "-I", str(SRC_DIR), "-c", str(src), "-o", str(obj)]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise BuildError(f"nvcc failed on {src.name}:\n{r.stdout}\n{r.stderr}")


def build_library(kind: str, head_dim=None, verbose: bool = True) -> Path:
    """Return the path of the library, compiling it first if it is not there."""
    target, sources, defines = library_path(kind, head_dim)
    if target.is_file():
        return target
    nvcc = find_nvcc()
    lock_path = target.with_suffix(".lock")
    with open(lock_path, "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)  # one builder at a time per library
        try:
            if target.is_file():
                return target
            t0 = time.time()
            if verbose:
                _say(f"compiling {target.name} from {len(sources)} sources for sm_100a (first use; a minute or so)")
            work = Path(tempfile.mkdtemp(prefix="krk_obj_", dir=str(target.parent)))
            stop = threading.Event()

            def ticker():
                while not stop.wait(10.0):
                    _say(f"  still compiling {target.name} ... {time.time() - t0:.0f}s")

            tick = threading.Thread(target=ticker, daemon=True)
            if verbose:
                tick.start()
            try:
                objs = [work / (Path(s).stem + ".o") for s in sources]
                with ThreadPoolExecutor(max_workers=min(8, len(sources))) as pool:
                    list(pool.map(lambda so: _compile_one(nvcc, SRC_DIR / so[0], so[1], defines), zip(sources, objs)))
                tmp = work / target.name
                libs = []
                if kind == "core":  # the library's directory as a run path too, should the process not hold a copy yet
                    lib_dir = Path(nvcc).resolve().parent.parent / "lib64"
                    libs = [f"-L{lib_dir}", *CORE_LIBS, "-Xlinker", f"-rpath={lib_dir}"]
                r = subprocess.run([nvcc, "-shared", "-o", str(tmp), *map(str, objs), "-gencode",
                                    "arch=compute_100a,code=sm_100a", *libs], capture_output=True, text=True)
                if r.returncode != 0:
                    raise BuildError(f"linking {target.name} failed:\n{r.stdout}\n{r.stderr}")
                os.replace(tmp, target)
            finally:
                stop.set()
                shutil.rmtree(work, ignore_errors=True)
            if verbose:
                _say(f"built {target.name} in {time.time() - t0:.1f}s")
            return target
        finally:
            fcntl.flock(lock, fcntl.LOCK_UN)
            try:
                os.unlink(lock_path)
            except OSError:
                pass


def build_all(head_dims=(16, 32, 64, 128), verbose: bool = True, latent_dims=((192, 128),)) -> list[Path]:
    """Compile the core library, the attention library of every given head size and the latent library of every given
    pair of sizes."""
    out = [build_library("core", verbose=verbose)] + [build_library(kind, verbose=verbose) for kind in SMALL_LIBRARIES]
    for d in head_dims:
        out.append(build_library("attn", d, verbose=verbose))
    for pair in latent_dims:
        out.append(build_library("latent", pair, verbose=verbose))
    return out
