"""Loader and builder for the native libraries.

``libats_b200.so`` holds every sm_100a kernel (plain C ABI, called through ctypes so that no
torch C++ headers are needed to build it and a launch costs a few microseconds of host time).
``libats_host.so`` holds the host-side C++ pieces (AVX CPU AdamW, data packing).  Both are built
in-tree under ``adaptivetrainingsystem_b200/_C`` with ``nvcc`` / ``g++``.

On a machine with a GPU a missing or stale CUDA library is an error, never a silent fallback.
"""
from __future__ import annotations

import ctypes
import glob
import os
import shutil
import subprocess
import threading
from concurrent.futures import ThreadPoolExecutor
from typing import List, Optional, Sequence

import torch

_PKG = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_ROOT = os.path.dirname(_PKG)
CSRC = os.path.join(_ROOT, "csrc")
OUT_DIR = os.path.join(_PKG, "_C")
CUDA_LIB = os.path.join(OUT_DIR, "libats_b200.so")
# the same kernels with every data-dependent index range-checked (-DATS_DEBUG); loaded instead of the release library when the
# environment says ATS_DEBUG_BUILD=1
DEBUG_LIB = os.path.join(OUT_DIR, "libats_b200_debug.so")
DEBUG_BUILD = os.environ.get("ATS_DEBUG_BUILD", "0") == "1"
HOST_LIB = os.path.join(OUT_DIR, "libats_host.so")

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden"]
# Every source is compiled with --use_fast_math except these: their kernels also serve models that run in true 32-bit.
PRECISE_MATH = {"dyt.cu", "latent_attention.cu", "delta_rule.cu", "channel_delta.cu", "lightning.cu", "gqa_attention.cu", "postnorm.cu"}
# Kernels that may only run in single-GPU jobs (none at present) would be listed here and built into a
# separate library so the main one never names a multicast load.
SINGLE_GPU_ONLY: List[str] = []

_lock = threading.Lock()
_cuda = None
_host = None


def _nvcc() -> Optional[str]:
    for cand in (shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    return None


def _stale(target: str, sources: List[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(s) > t for s in sources)


def cuda_sources() -> List[str]:
    return sorted(s for s in glob.glob(os.path.join(CSRC, "*.cu")) if os.path.basename(s) not in SINGLE_GPU_ONLY)


def _nvcc_or_raise() -> str:
    nvcc = _nvcc()
    if nvcc is None:
        raise RuntimeError("nvcc not found; cannot build the sm_100a kernels")
    return nvcc


def _compile_objects(srcs: List[str], tag: str, extra: List[str], force: bool, verbose: bool = False) -> List[str]:
    """One object per source under ``_C/obj_<tag>``, compiled in parallel; up-to-date objects are kept."""
    nvcc = _nvcc_or_raise()
    headers = glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h"))
    obj_dir = os.path.join(OUT_DIR, f"obj_{tag}")
    os.makedirs(obj_dir, exist_ok=True)

    def one(src: str) -> str:
        obj = os.path.join(obj_dir, os.path.basename(src)[:-3] + ".o")
        if not (force or _stale(obj, [src] + headers)):
            return obj
        math = [] if os.path.basename(src) in PRECISE_MATH else ["--use_fast_math"]
        cmd = [nvcc] + NVCC_FLAGS + math + extra + ["-I", CSRC, "-c", "-o", obj + ".tmp.o", src]
        if verbose:
            cmd[1:1] = ["-Xptxas", "-v"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed on {os.path.basename(src)}:\n" + r.stdout + r.stderr)
        if verbose:
            print(r.stderr)
        os.replace(obj + ".tmp.o", obj)
        return obj
    with ThreadPoolExecutor(max_workers=min(len(srcs), os.cpu_count() or 4)) as pool:
        return list(pool.map(one, srcs))


def _link(target: str, objects: List[str], extra: List[str]) -> None:
    cmd = [_nvcc_or_raise()] + NVCC_FLAGS + extra + ["-shared", "-o", target + ".tmp"] + objects
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("nvcc (link) failed:\n" + r.stdout + r.stderr)
    os.replace(target + ".tmp", target)


def _build_library(target: str, srcs: List[str], tag: str, extra: List[str], force: bool, verbose: bool = False) -> None:
    headers = glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h"))
    if force or _stale(target, srcs + headers):
        _link(target, _compile_objects(srcs, tag, extra, force, verbose), extra)


def build_debug(force: bool = False) -> None:
    """The bounds-checking build: -DATS_DEBUG, relocatable device code (one report word shared by all translation units)."""
    os.makedirs(OUT_DIR, exist_ok=True)
    _build_library(DEBUG_LIB, cuda_sources(), "debug", ["-DATS_DEBUG", "-rdc=true"], force)


def build(force: bool = False, verbose: bool = False) -> None:
    """Compile every native source for sm_100a (cross-compiles without a GPU)."""
    os.makedirs(OUT_DIR, exist_ok=True)
    extra = os.environ.get("ATS_NVCC_EXTRA", "").split()  # e.g. -DATS_AB_SPLIT=4 for kernel tuning experiments
    _build_library(CUDA_LIB, cuda_sources(), "release", extra, force, verbose)
    host_srcs = sorted(glob.glob(os.path.join(CSRC, "host", "*.cpp")))
    if host_srcs and (force or _stale(HOST_LIB, host_srcs)):
        cxx = shutil.which("g++") or "g++"
        cmd = [cxx, "-O3", "-std=c++17", "-fPIC", "-shared", "-fopenmp", "-mavx2", "-mfma", "-o", HOST_LIB + ".tmp"] + host_srcs
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("g++ failed:\n" + r.stdout + r.stderr)
        os.replace(HOST_LIB + ".tmp", HOST_LIB)


def load_for(sources: Sequence[str], name: str) -> ctypes.CDLL:
    """The kernel library for a program that serves one model: the full library when it has been built, otherwise a library of
    only the named ``csrc`` files (``libats_<name>.so``), so that a fresh checkout compiles what the model needs and no more."""
    global _cuda
    with _lock:
        if _cuda is None and not DEBUG_BUILD and not os.path.exists(CUDA_LIB):
            part = os.path.join(OUT_DIR, f"libats_{name}.so")
            os.makedirs(OUT_DIR, exist_ok=True)
            _build_library(part, [os.path.join(CSRC, s) for s in sources], "release", [], False)
            _cuda = ctypes.CDLL(part)
    return cuda_lib()


def cuda_lib() -> ctypes.CDLL:
    """The CUDA kernel library; raises if it is not there."""
    global _cuda
    if _cuda is None:
        with _lock:
            if _cuda is None:
                path = DEBUG_LIB if DEBUG_BUILD else CUDA_LIB
                if not os.path.exists(path):
                    if _nvcc() is not None:
                        build_debug() if DEBUG_BUILD else build()
                    else:
                        raise RuntimeError(f"{path} is missing and nvcc is unavailable; run __graft_entry__.build()")
                _cuda = ctypes.CDLL(path)
    return _cuda


def host_lib() -> Optional[ctypes.CDLL]:
    global _host
    if _host is None:
        with _lock:
            if _host is None:
                if not os.path.exists(HOST_LIB):
                    try:
                        build()
                    except Exception:
                        return None
                if os.path.exists(HOST_LIB):
                    _host = ctypes.CDLL(HOST_LIB)
    return _host


def use_cuda_kernels(t: torch.Tensor) -> bool:
    """Kernels take bf16 CUDA tensors; everything else (CPU, fp32 oracles) runs the PyTorch definition."""
    return t.is_cuda and t.dtype == torch.bfloat16 and os.environ.get("ATS_FORCE_TORCH", "0") != "1"


class KernelError(RuntimeError):
    pass


_STATUS_NAMES = {1: "TMA stage never arrived", 2: "TMA stage never released", 3: "accumulator never produced",
                 4: "accumulator never released", 5: "peer flag never arrived", 6: "bad argument"}
_DEBUG_KERNELS = {1: "plan_slots", 2: "dispatch_rows", 3: "combine_rows", 4: "slot_dot", 5: "grouped GEMM row counts", 6: "decode attention",
                  7: "serve_plan_dispatch", 8: "serve_combine", 9: "embedding_bwd", 10: "peer_reduce", 11: "mod_rows"}


def debug_report() -> Optional[dict]:
    """Debug build only: the first failed bounds check since the last call ({kernel, block, detail}), or ``None``; clears it."""
    if not DEBUG_BUILD or _cuda is None:
        return None
    out = (ctypes.c_int * 4)()
    _cuda.ats_debug_report.restype = ctypes.c_int
    _cuda.ats_debug_report.argtypes = [ctypes.POINTER(ctypes.c_int)]
    if _cuda.ats_debug_report(out) != 1 or out[0] == 0:
        return None
    return {"code": out[0], "kernel": _DEBUG_KERNELS.get(out[1], out[1]), "block": out[2], "detail": out[3]}
_status = {}


def status_tensor(device: torch.device) -> torch.Tensor:
    """One int32 word per device that kernels set when a bounded wait runs out."""
    key = torch.device(device).index or 0
    if key not in _status:
        _status[key] = torch.zeros(4, dtype=torch.int32, device=device)
    return _status[key]


def check_status(device=None) -> None:
    """Raise if any kernel reported a timed-out wait (synchronises the device)."""
    for key, t in list(_status.items()):
        v = int(t[0].item())
        if v != 0:
            t.zero_()
            raise KernelError(f"device {key}: kernel wait timed out: {_STATUS_NAMES.get(v, v)}")
    rep = debug_report()
    if rep is not None:
        raise KernelError(f"bounds check failed in {rep['kernel']} (block {rep['block']}, value {rep['detail']}); the access was skipped")


_launches = 0


def launch_count() -> int:
    """Number of native entry points called so far (each launches at least one kernel)."""
    return _launches


def check(err: int, what: str) -> None:
    global _launches
    _launches += 1
    if err != 0:
        if err >= 1000:
            raise KernelError(f"{what}: argument/tensor-map error {err}")
        raise KernelError(f"{what}: CUDA error {err}")


def ptr(t: Optional[torch.Tensor]) -> ctypes.c_void_p:
    return ctypes.c_void_p(0 if t is None else t.data_ptr())


def stream_ptr(device=None) -> ctypes.c_void_p:
    return ctypes.c_void_p(torch.cuda.current_stream(device).cuda_stream)
