"""Builds the C-ABI library in-tree with nvcc for sm_100a.

Run as `python -m minivllm_b200.csrc.build` for libminivllm_b200.so with every kernel.  The package never builds at
import time.  Programs that must work from a fresh checkout call `build(group=...)`: it compiles only the sources one
model family needs into a library of its own, and does nothing when the full library is there and up to date.
"""
import contextlib
import fcntl
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
LIB = os.path.join(HERE, "libminivllm_b200.so")
COMMON = ["api.cu", "metadata.cu", "sampling.cu"]
GROUPS = {
    "qwen3": ["store_kvcache.cu", "paged_decode.cu", "paged_decode_int8.cu", "prefill_varlen.cu",
              "paged_decode_static.cu", "pre_attention.cu", "comm.cu"],
    "sipazen": ["norms.cu", "latent_attention.cu", "latent_decode.cu", "latent_prefill.cu", "short_conv.cu", "mamba2.cu",
                "mamba2_chunk.cu", "moe.cu", "grouped_gemm.cu"],
    "fozerax": ["norms.cu", "window_attention.cu", "latent_prefill.cu", "short_conv.cu", "gla.cu", "gla_chunk.cu", "gated_delta.cu",
                "gated_delta_chunk.cu", "moe.cu", "grouped_gemm.cu"],
    "dafotar": ["norms.cu", "streams.cu", "short_conv.cu", "window_attention.cu", "latent_prefill.cu", "mlstm.cu", "mlstm_chunk.cu"],
    "subivik": ["norms.cu", "tanh_norm.cu", "short_conv.cu", "window_attention.cu", "latent_prefill.cu", "talk_attention.cu",
                "talk_prefill.cu", "time_mix.cu", "gla_chunk.cu", "moe.cu", "grouped_gemm.cu"],
}
SOURCES = COMMON + list(dict.fromkeys(s for g in GROUPS.values() for s in g))
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]


def group_lib(group):
    return os.path.join(HERE, f"libminivllm_b200_{group}.so")


def _stale(target, deps):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


@contextlib.contextmanager
def _lock():
    """One build at a time in a checkout."""
    with open(os.path.join(HERE, ".build.lock"), "w") as f:
        fcntl.flock(f, fcntl.LOCK_EX)
        yield


def build(verbose=False, force=False, group=None):
    """Returns the path of an up-to-date library: the full one, or with `group` one that serves that family."""
    headers = [os.path.join(HERE, f) for f in os.listdir(HERE) if f.endswith((".cuh", ".h"))]
    headers.append(os.path.join(HERE, "..", "..", "include", "minivllm_b200.h"))
    path = lambda names: [os.path.join(HERE, s) for s in names]
    if group is not None:
        if not _stale(LIB, path(SOURCES) + headers):
            return LIB
        lib, sources = group_lib(group), COMMON + GROUPS[group]
        if not force and not _stale(lib, path(sources) + headers):
            return lib
    else:
        lib, sources = LIB, SOURCES
    with _lock():
        return _build(lib, sources, headers, verbose, force)


def _build(lib, sources, headers, verbose, force):
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    objs, jobs = [], []
    for src in sources:
        s = os.path.join(HERE, src)
        o = os.path.join(HERE, src.replace(".cu", ".o"))
        objs.append(o)
        if force or _stale(o, [s] + headers):
            cmd = [nvcc] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", s, "-o", o]
            if verbose:
                print(" ".join(cmd), file=sys.stderr, flush=True)
            jobs.append(cmd)
    if jobs:
        with ThreadPoolExecutor(max_workers=min(len(jobs), os.cpu_count() or 1)) as pool:
            list(pool.map(lambda c: subprocess.check_call(c, stdout=sys.stderr), jobs))
    if force or _stale(lib, objs):
        part = lib + ".part"
        cmd = [nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "-shared", "-o", part] + objs + ["-lcudart"]
        if verbose:
            print(" ".join(cmd), file=sys.stderr, flush=True)
        subprocess.check_call(cmd, stdout=sys.stderr)
        os.replace(part, lib)
    return lib


if __name__ == "__main__":
    build(verbose="-v" in sys.argv, force="-f" in sys.argv)
    print(LIB)
