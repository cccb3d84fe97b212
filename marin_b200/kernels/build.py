"""Compiles the CUDA sources of ``csrc/`` for sm_100a (and the C++ host sources of ``csrc/host/``) into shared
libraries, at first use.

Each library is built with ``nvcc`` directly (no framework headers, so a file compiles in
seconds) into ``marin_b200/csrc/_build/`` beside the sources, named by a hash of its sources
and flags, and loaded with ``ctypes``.  The reference compiles its kernels at start-up too
(NVRTC, crates/cuda/src/gpu.rs:159-164).  If the package folder is read-only the build goes to
a per-user temporary folder.  A line is printed when a compile starts and every few seconds
while it runs, so that a first call does not look hung.
"""
from __future__ import annotations

import ctypes
import hashlib
import os
import shutil
import subprocess
import sys
import tempfile
import threading
import time
from typing import Dict, List, Optional, Sequence

CSRC = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "csrc")
ARCH_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a"]
BASE_FLAGS = ["-O3", "-std=c++17", "-lineinfo", "--shared", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden"]

_loaded: Dict[str, ctypes.CDLL] = {}
_lock = threading.Lock()


class KernelBuildError(RuntimeError):
    pass


def _nvcc() -> str:
    for cand in (os.environ.get("MARIN_B200_NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise KernelBuildError("nvcc was not found (looked at $MARIN_B200_NVCC, PATH and /usr/local/cuda/bin); "
                           "the CUDA kernels of marin_b200 cannot be built and there is no other path")


HOST_FLAGS = ["-O2", "-std=c++17", "-shared", "-fPIC", "-fvisibility=hidden"]


def _host_compiler() -> str:
    for cand in (os.environ.get("CXX"), shutil.which("g++"), shutil.which("c++"), shutil.which("clang++")):
        if cand and (os.path.exists(cand) or shutil.which(cand)):
            return cand
    raise KernelBuildError("no C++ compiler was found (looked at $CXX, g++, c++, clang++): the host code of marin_b200 cannot be built")


def _is_host(sources: Sequence[str]) -> bool:
    return all(s.endswith(".cpp") for s in sources)


_build_dir_cache: Optional[str] = None
_dir_lock = threading.Lock()


def _build_dir() -> str:
    global _build_dir_cache
    with _dir_lock:
        if _build_dir_cache is not None:
            return _build_dir_cache
        override = os.environ.get("MARIN_B200_BUILD_DIR")
        candidates = [override] if override else []
        candidates.append(os.path.join(CSRC, "_build"))
        candidates.append(os.path.join(tempfile.gettempdir(), f"marin_b200_build_{os.getuid()}"))
        for path in candidates:
            try:
                os.makedirs(path, exist_ok=True)
                fd, probe = tempfile.mkstemp(prefix=".probe", dir=path)
                os.close(fd)
                os.remove(probe)
                _build_dir_cache = path
                return path
            except OSError:
                continue
        raise KernelBuildError(f"no writable build folder among {candidates}")


def _digest(sources: Sequence[str], flags: Sequence[str]) -> str:
    h = hashlib.sha256()
    folders = sorted({""} | {os.path.dirname(s) for s in sources})       # headers beside the sources count too
    for folder in folders:
        for name in sorted(os.listdir(os.path.join(CSRC, folder))):
            if name.endswith((".cuh", ".h")):
                with open(os.path.join(CSRC, folder, name), "rb") as fh:
                    h.update(os.path.join(folder, name).encode() + b"\0" + fh.read())
    for src in sources:
        with open(os.path.join(CSRC, src), "rb") as fh:
            h.update(src.encode() + b"\0" + fh.read())
    h.update(" ".join(flags).encode())
    return h.hexdigest()[:16]


def library_path(name: str, sources: Sequence[str], defines: Sequence[str] = ()) -> str:
    flags = ARCH_FLAGS + BASE_FLAGS + [f"-D{d}" for d in defines]
    return os.path.join(_build_dir(), f"{name}-{_digest(sources, flags)}.so")


def build(name: str, sources: Sequence[str], defines: Sequence[str] = (), verbose: bool = True) -> str:
    """Compiles ``sources`` (names inside csrc/) into one shared library unless it is already built.
    MARIN_B200_DEFINES in the environment (comma separated, e.g. ``DEC_STAGES=2,PDL_WAIT_FIRST``) adds defines to
    every library: the kernels' tuning constants can be overridden for experiments without touching the sources."""
    extra = [x for x in os.environ.get("MARIN_B200_DEFINES", "").split(",") if x]
    host = _is_host(sources)
    flags = (HOST_FLAGS if host else ARCH_FLAGS + BASE_FLAGS) + [f"-D{d}" for d in list(defines) + extra]
    out = os.path.join(_build_dir(), f"{name}-{_digest(sources, flags)}.so")
    if os.path.exists(out):
        return out
    tmp = f"{out}.{os.getpid()}.{threading.get_ident()}.tmp"
    cmd = [_host_compiler() if host else _nvcc()] + flags + ["-I", CSRC, "-o", tmp] + [os.path.join(CSRC, s) for s in sources]
    if verbose:
        print(f"[marin_b200] compiling {name} {'(host code)' if host else 'for sm_100a'} ({', '.join(sources)}) ...", file=sys.stderr, flush=True)
    started = time.time()
    proc = subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    while True:
        try:
            output, _ = proc.communicate(timeout=10)
            break
        except subprocess.TimeoutExpired:
            if verbose:
                print(f"[marin_b200] ... still compiling {name} ({time.time() - started:.0f} s)", file=sys.stderr, flush=True)
    if proc.returncode != 0:
        if os.path.exists(tmp):
            os.remove(tmp)
        raise KernelBuildError(f"nvcc failed for {name}:\n{' '.join(cmd)}\n{output}")
    os.replace(tmp, out)
    if verbose:
        print(f"[marin_b200] built {os.path.basename(out)} in {time.time() - started:.1f} s", file=sys.stderr, flush=True)
    return out


def load(name: str, sources: Sequence[str], defines: Sequence[str] = ()) -> ctypes.CDLL:
    """The library, built if need be and loaded once per process."""
    key = name + "|" + "|".join(defines)
    with _lock:
        lib = _loaded.get(key)
        if lib is None:
            lib = ctypes.CDLL(build(name, sources, defines))
            _loaded[key] = lib
        return lib


#: every library of the package: name → sources.  ``build_all`` compiles them all.
LIBRARIES: Dict[str, List[str]] = {
    "mb_elementwise": ["elementwise.cu"],
    "mb_gemm_simple": ["gemm_simple.cu"],
    "mb_attention_simple": ["attention_simple.cu"],
    "mb_sampling": ["sampling.cu"],
    "mb_gemm_tc": ["gemm_tc.cu"],
    "mb_activations": ["activations.cu"],
    "mb_recurrent": ["recurrent.cu"],
    "mb_attention_sigmoid": ["attention_sigmoid.cu"],
    "mb_hyper": ["hyper.cu"],
    "mb_attention_sink": ["attention_sink.cu"],
    "mb_attention_latent": ["attention_latent.cu"],
    "mb_moe": ["moe.cu"],
    "mb_attention_pooled": ["attention_pooled.cu"],
    "mb_ssm": ["ssm.cu"],
    "mb_layer_norm": ["layer_norm.cu"],
    "mb_delta_rule": ["delta_rule.cu"],
    "mb_gated_linear": ["gated_linear.cu"],
    "mb_host": ["host/cache_core.cpp", "host/scheduler.cpp", "host/sampler.cpp", "host/safetensors.cpp"],
}


#: (head size, query heads per kv head) the fast attention kernels are built for by ``build_all``; any other
#: layout a model brings is compiled when that model first runs
ATTENTION_LAYOUTS = [(128, 4), (128, 5), (128, 2), (16, 2), (32, 4), (48, 2)]
#: (page row, latent width, query heads) of attention over a shared latent the tcgen05 prompt kernel is built for by ``build_all``
LATENT_LAYOUTS = [(160, 128, 32), (80, 64, 8)]


def build_many(jobs: Dict[str, tuple], verbose: bool = True) -> List[str]:
    """Compiles ``{name: (sources, defines)}`` in parallel; returns the libraries' paths."""
    results: Dict[str, object] = {}

    def work(n: str) -> None:
        try:
            results[n] = build(n, jobs[n][0], jobs[n][1], verbose=verbose)
        except Exception as err:  # noqa: BLE001 - reported below
            results[n] = err

    threads = [threading.Thread(target=work, args=(n,)) for n in jobs]
    for t in threads:
        t.start()
    for t in threads:
        t.join()
    errors = [r for r in results.values() if isinstance(r, Exception)]
    if errors:
        raise errors[0]
    return [str(results[n]) for n in jobs]


def attention_job(d: int, group: int) -> tuple:
    """Sources and defines of the attention kernels for one head layout."""
    return (["attention_fast.cu"], [f"HEAD_DIM={d}", f"GROUP={group}"])


def attention_tc_job(d: int, group: int, dv: int = 0, values_in_keys: bool = False, pair: bool = False) -> tuple:
    """Sources and defines of the tensor-core prefill attention kernel for one head layout (``dv`` 0: values as wide as the keys;
    ``values_in_keys``: the values are the first ``dv`` elements of the key rows; ``pair``: query heads are pairs of maps)."""
    if values_in_keys:
        return (["attention_tc.cu"], [f"HEAD_DIM={d}", f"V_DIM={dv}", f"GROUP={group}", "V_IN_K"])
    return (["attention_tc.cu"], [f"HEAD_DIM={d}", f"GROUP={group}"] + ([f"V_DIM={dv}"] if dv not in (0, d) else []) + (["PAIR"] if pair else []))


def attention_tc_name(d: int, group: int, dv: int = 0, values_in_keys: bool = False, pair: bool = False) -> str:
    if values_in_keys:
        return f"mb_attention_tc_d{d}_v{dv}_g{group}_vk"
    return f"mb_attention_tc_d{d}" + (f"_v{dv}" if dv not in (0, d) else "") + f"_g{group}" + ("_pair" if pair else "")


#: One or two layouts of every source that is otherwise compiled for a model's own sizes when it first runs (the names and
#: defines are those the wrappers in ``ops`` use): sink attention with keys and values of their own and over a shared latent
#: with sixteen heads a CTA, sigmoid attention, chunked linear attention, attention over a window and pooled blocks, the chunked
#: delta rule, chunked gated linear attention, two maps per head.
PER_LAYOUT_SAMPLES = {
    "mb_attention_sink_fast_d128_v128_g4": (["attention_sink_fast.cu"], ["HEAD_DIM=128", "V_DIM=128", "GROUP=4"]),
    "mb_attention_sink_fast_d160_v128_g16_vk": (["attention_sink_fast.cu"], ["HEAD_DIM=160", "V_DIM=128", "GROUP=16", "V_IN_K"]),
    "mb_attention_sigmoid_fast_d128_v128_g4": (["attention_sigmoid_fast.cu"], ["HEAD_DIM=128", "V_DIM=128", "GROUP=4"]),
    "mb_linear_attention_chunked_d128_v32": (["linear_attention_chunked.cu"], ["QK_DIM=128", "V_SLICE=32"]),
    "mb_delta_rule_chunked_d128_v32": (["delta_rule_chunked.cu"], ["QK_DIM=128", "V_SLICE=32"]),
    "mb_gated_linear_chunked_d128_v128": (["gated_linear_chunked.cu"], ["QK_DIM=128", "V_SLICE=128"]),
    "mb_attention_sink_fast_d128_v128_g8": (["attention_sink_fast.cu"], ["HEAD_DIM=128", "V_DIM=128", "GROUP=8"]),
    "mb_attention_tc_d128_g8_pair": (["attention_tc.cu"], ["HEAD_DIM=128", "GROUP=8", "PAIR"]),
    "mb_attention_pooled_fast_d128_v128_g4_c2": (["attention_pooled_fast.cu"], ["HEAD_DIM=128", "V_DIM=128", "GROUP=4", "VALUE_HEADS=2"]),
}


def build_all(verbose: bool = True) -> List[str]:
    """Compiles every library and the attention kernels for the layouts in ``ATTENTION_LAYOUTS`` (in parallel).
    Used by the build check and before timing."""
    jobs = {n: (src, []) for n, src in LIBRARIES.items()}
    for d, g in ATTENTION_LAYOUTS:
        jobs[f"mb_attention_fast_d{d}_g{g}"] = attention_job(d, g)
        if d in (64, 128):
            jobs[f"mb_attention_tc_d{d}_g{g}"] = attention_tc_job(d, g)
    for d, dv, g in LATENT_LAYOUTS:
        jobs[attention_tc_name(d, g, dv, True)] = attention_tc_job(d, g, dv, True)
    jobs.update(PER_LAYOUT_SAMPLES)
    return build_many(jobs, verbose)


def build_for(model, dtype, verbose: bool = True) -> List[str]:
    """Compiles what this model needs and nothing else: the element-wise and sampling kernels, the matrix products of
    its dtype, and whatever its parts ask for themselves (``Part.kernel_jobs``: attention for its head layouts)."""
    import torch

    jobs = {"mb_elementwise": (LIBRARIES["mb_elementwise"], []), "mb_sampling": (LIBRARIES["mb_sampling"], []),
            "mb_gemm_simple": (LIBRARIES["mb_gemm_simple"], [])}
    if dtype == torch.bfloat16:
        jobs["mb_gemm_tc"] = (LIBRARIES["mb_gemm_tc"], [])
    if hasattr(model, "kernel_jobs"):
        jobs.update(model.kernel_jobs(dtype))
    return build_many(jobs, verbose)
