"""In-tree build of the native libraries.

Three shared objects are produced next to this file:

* ``_C_core.so``  the kernels of ``CORE_SOURCES`` + ``csrc/bindings_core.cpp``: matrix products, MoE
                  routing, sampling, gated / windowed attention, the 32-bit residual stream.  Some
                  models run on this library alone (``ensure_core`` builds nothing else).
* ``_C.so``       all other CUDA kernels for sm_100a (``csrc/**/*.cu``) + ``csrc/bindings.cpp``,
                  linked against ``_C_core.so``.  Both register ``torch.ops.omni_b200.*``.
* ``_runtime.so`` host-only C++ runtime pieces (``csrc/runtime``, ``csrc/alloc``):
                  KV block allocator, scheduler helpers, VMM sleep-mode allocator.

Kernels are compiled one translation unit per ``.cu`` file with
``nvcc -gencode arch=compute_100a,code=sm_100a`` (no torch headers in device
code, so a file builds in seconds) and linked together with the bindings,
which are compiled by the host compiler against the torch headers.  Objects are
rebuilt only when their source (or a header) is newer.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
OBJ = PKG.parent / "build" / "obj"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--use_fast_math", "-Xcompiler", "-fPIC", "-Xptxas", "-v",
]
CXX_FLAGS = ["-O2", "-std=c++17", "-fPIC", "-Wall", "-Wno-unused-function"]


# sources of the core library, relative to csrc/
CORE_SOURCES = [
    "attn/gqa_gated.cu", "attn/gqa_gated_decode.cu", "attn/gqa_gated_prefill.cu", "attn/gqa_prefill_tcgen05.cu",
    "attn/latent_attn.cu", "attn/mixed_attn.cu", "attn/mixed_attn_decode.cu", "attn/mixed_attn_prefill.cu",
    "attn/mla_decode.cu", "attn/qk_norm_rope.cu",
    "gemm/gemm_simt.cu", "gemm/gemm_tcgen05.cu", "gemm/gemm_tcgen05_pair.cu", "moe/moe_ep.cu",
    "norm_rope/hyper_norm.cu", "norm_rope/post_norm.cu", "norm_rope/residual_norm.cu", "recurrent/decay_prep.cu", "recurrent/recurrent.cu",
    "sample/sampling.cu",
]

# sources whose fp32 functions and divisions keep their full accuracy
PRECISE_SOURCES = ["attn/latent_attn.cu", "attn/mixed_attn.cu", "attn/qk_norm_rope.cu", "gemm/gemm_simt.cu",
                   "norm_rope/hyper_norm.cu", "norm_rope/post_norm.cu", "recurrent/decay_prep.cu", "recurrent/recurrent.cu"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", shutil.which("nvcc")):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


def _cuda_home() -> str:
    return str(Path(_nvcc()).resolve().parent.parent)


def _newest_header_mtime() -> float:
    m = 0.0
    for ext in ("*.cuh", "*.h", "*.hpp"):
        for p in CSRC.rglob(ext):
            m = max(m, p.stat().st_mtime)
    return m


def _stale(src: Path, obj: Path, hdr_mtime: float) -> bool:
    if not obj.exists():
        return True
    t = obj.stat().st_mtime
    return src.stat().st_mtime > t or hdr_mtime > t or Path(__file__).stat().st_mtime > t


def _run(cmd: list[str], log: Path | None = None) -> None:
    r = subprocess.run(cmd, capture_output=True, text=True)
    if log is not None:
        log.write_text(r.stdout + r.stderr)
    if r.returncode != 0:
        raise RuntimeError("command failed: %s\n%s\n%s" % (" ".join(cmd), r.stdout, r.stderr))


def cuda_sources() -> list[Path]:
    return sorted(p for p in CSRC.rglob("*.cu"))


def runtime_sources() -> list[Path]:
    out: list[Path] = []
    for d in ("runtime", "alloc"):
        out += sorted((CSRC / d).glob("*.cpp"))
    return out


def core_is_current() -> bool:
    """Whether ``_C_core.so`` exists and is newer than everything it is made of."""
    lib = PKG / "_C_core.so"
    if not lib.exists():
        return False
    t = lib.stat().st_mtime
    srcs = [CSRC / x for x in CORE_SOURCES] + [CSRC / "bindings_core.cpp"]
    return all(p.stat().st_mtime <= t for p in srcs) and _newest_header_mtime() <= t


def ensure_core(verbose: bool = False) -> None:
    """Build the core library alone when it is missing or older than its sources (one process at a
    time; the others wait for it)."""
    if core_is_current():
        return
    import fcntl
    OBJ.mkdir(parents=True, exist_ok=True)
    with open(OBJ / ".lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not core_is_current():
            build(verbose=verbose, core_only=True)


def build(force: bool = False, verbose: bool = False, core_only: bool = False) -> dict:
    """Compile everything that is out of date (``core_only``: for the core library alone).  Returns
    the paths of the libraries."""
    import sysconfig

    import torch  # (import first: the headers' location comes from it)
    from torch.utils import cpp_extension as ce

    OBJ.mkdir(parents=True, exist_ok=True)
    hdr_mtime = _newest_header_mtime()
    nvcc = _nvcc()
    cuda_home = _cuda_home()
    jobs: list[tuple[list[str], Path | None]] = []
    objs: dict[str, list[Path]] = {"_C_core": [], "_C": [], "_runtime": []}
    dirty: set[str] = set()

    def compile_one(src: Path, lib: str, cmd: list[str], log: bool = False) -> None:
        obj = OBJ / (src.relative_to(CSRC).as_posix().replace("/", "__") + ".o")
        objs[lib].append(obj)
        if force or _stale(src, obj, hdr_mtime):
            dirty.add(lib)
            jobs.append(([*cmd, "-c", str(src), "-o", str(obj)], obj.with_suffix(".log") if log else None))

    for src in cuda_sources():
        lib = "_C_core" if src.relative_to(CSRC).as_posix() in CORE_SOURCES else "_C"
        flags = NVCC_FLAGS
        if src.relative_to(CSRC).as_posix() in PRECISE_SOURCES:
            flags = [f for f in flags if f != "--use_fast_math"]
        if lib == "_C_core" or not core_only:
            compile_one(src, lib, [nvcc, *flags, "-I", str(CSRC)], log=True)

    inc = []
    for p in ce.include_paths("cuda") if hasattr(ce, "include_paths") else []:
        inc += ["-I", p]
    inc += ["-I", os.path.join(cuda_home, "include"), "-I", sysconfig.get_paths()["include"]]
    abi = int(getattr(torch._C, "_GLIBCXX_USE_CXX11_ABI", 1))
    cxx = ["g++", *CXX_FLAGS, f"-D_GLIBCXX_USE_CXX11_ABI={abi}", *inc]
    compile_one(CSRC / "bindings_core.cpp", "_C_core", cxx)
    if not core_only:
        compile_one(CSRC / "bindings.cpp", "_C", cxx)
        for src in runtime_sources():
            compile_one(src, "_runtime", ["g++", *CXX_FLAGS, "-I", os.path.join(cuda_home, "include"), "-I", str(CSRC)])

    if jobs:
        if verbose:
            print(f"[omni_npu_b200] compiling {len(jobs)} translation units", file=sys.stderr)
        with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 4)) as ex:
            list(ex.map(lambda j: _run(j[0], j[1]), jobs))

    torch_lib = os.path.join(os.path.dirname(torch.__file__), "lib")
    libs = ["-lc10", "-ltorch_cpu", "-ltorch", "-lc10_cuda", "-ltorch_cuda", f"-L{cuda_home}/lib64", "-lcudart",
            f"-Wl,-rpath,{torch_lib}", f"-Wl,-rpath,{cuda_home}/lib64"]

    def link(name: str, extra: list[str]) -> Path:
        out = PKG / f"{name}.so"
        if name in dirty or not out.exists():
            part = out.with_suffix(f".so.{os.getpid()}")      # in place in one step: others may be loading it
            _run(["g++", "-shared", "-o", str(part), f"-Wl,-soname,{out.name}", *map(str, objs[name]), *extra])
            os.replace(part, out)
        return out

    out = {"_C_core": link("_C_core", [f"-L{torch_lib}", *libs])}
    if not core_only:
        out["_C"] = link("_C", [f"-L{PKG}", "-l:_C_core.so", "-Wl,-rpath,$ORIGIN", f"-L{torch_lib}", *libs])
        out["_runtime"] = link("_runtime", ["-ldl", "-lpthread"]) if objs["_runtime"] else None
    return out


if __name__ == "__main__":
    out = build(force="--force" in sys.argv, verbose=True)
    print(out)
