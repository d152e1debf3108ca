"""In-tree native build: CUDA kernels (nvcc, sm_100a) and the C++ host core (g++, pybind11).

Both libraries are written next to the package (``skein_b200/_native``) so that a snapshot of the
source tree carries them along; nothing is installed into site-packages and nothing depends on a
JIT cache in the home directory.

    python -m skein_b200._build            # build whatever is out of date
    python -m skein_b200._build --force    # rebuild everything

`ensure_built(architecture)` compiles, in a fresh checkout, only the kernels that architecture's models run.
"""
from __future__ import annotations

import concurrent.futures as cf
import contextlib
import fcntl
import os
import shutil
import subprocess
import sys
import sysconfig
from pathlib import Path

ROOT = Path(__file__).resolve().parent.parent
CSRC = ROOT / "csrc"
NATIVE = Path(__file__).resolve().parent / "_native"
OBJ = ROOT / "build" / "obj"

KERNEL_LIB = NATIVE / "libskein_kernels.so"
CORE_LIB_STEM = "_skein_core"

# Kernel sources of architectures that need only some of them (the others take the whole library).
ARCH_SOURCES = {
    "Zarorax": ("attn_latent_decode", "attn_latent_prefill", "gemm_simt", "gemm_small", "gemm_ws", "latent", "postnorm", "rope_kv", "router", "sample"),
    "Sikalorn": ("attn_decode", "attn_decode_mma", "attn_prefill_tc", "attn_window", "gemm_simt", "gemm_small", "gemm_ws", "parallel_layer", "postnorm", "recurrent",
                 "recurrent_tc", "rope_kv", "sample"),
    "Barorax": ("attn_decode", "attn_decode_mma", "attn_prefill_tc", "attn_window", "gemm_simt", "gemm_small", "gemm_ws", "postnorm", "prenorm", "rope_kv", "router",
                "sample", "selective"),
    "Derusun": ("attn_decode", "attn_decode_mma", "attn_latent_decode", "attn_latent_prefill", "attn_prefill_tc", "attn_window", "gemm_simt", "gemm_small",
                "gemm_ws", "latent", "parallel_layer", "postnorm", "prenorm", "recurrent", "recurrent_channel_tc", "recurrent_tc", "rope_kv", "sample"),
}
# Sources compiled without fast-math: their exponentials, logarithms and tanh keep the accuracy of 32-bit.
EXACT_SOURCES = ("attn_window", "parallel_layer", "prenorm", "recurrent", "recurrent_channel_tc", "recurrent_tc", "selective")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "--use_fast_math", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=default",
]
CXX_FLAGS = ["-O2", "-std=c++17", "-fPIC", "-Wall", "-Wno-sign-compare", "-pthread"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found (set NVCC or put /usr/local/cuda/bin on PATH)")


def _newer(src: Path, dst: Path, extra_deps=()) -> bool:
    if not dst.exists():
        return True
    t = dst.stat().st_mtime
    return any(p.stat().st_mtime > t for p in (src, *extra_deps))


def _run(cmd):
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("command failed: %s\n%s\n%s" % (" ".join(map(str, cmd)), r.stdout, r.stderr))
    return r.stdout + r.stderr


def core_lib_path() -> Path:
    return NATIVE / (CORE_LIB_STEM + sysconfig.get_config_var("EXT_SUFFIX"))


@contextlib.contextmanager
def _locked():
    """One build at a time in a checkout."""
    NATIVE.mkdir(parents=True, exist_ok=True)
    OBJ.mkdir(parents=True, exist_ok=True)
    with open(OBJ / ".lock", "w") as f:
        fcntl.flock(f, fcntl.LOCK_EX)
        yield


def _link(cmd, out: Path) -> None:
    """Link beside the target and rename over it: a process that has the old library mapped keeps it."""
    tmp = out.with_name(f".{out.name}.{os.getpid()}")
    _run([*cmd[:2], "-o", str(tmp), *cmd[2:]])
    os.replace(tmp, out)


def build_kernels(force: bool = False, verbose: bool = False, only=None) -> Path:
    """Compile csrc/kernels/*.cu for sm_100a (all, or the stems in `only` besides those compiled before) and link
    libskein_kernels.so from what has been compiled."""
    kdir = CSRC / "kernels"
    headers = sorted(kdir.glob("*.cuh")) + sorted(kdir.glob("*.h"))
    srcs = [s for s in sorted(kdir.glob("*.cu")) if only is None or s.stem in only or (OBJ / (s.stem + ".o")).exists()]
    nvcc = _nvcc()
    jobs = []
    objs = []
    for s in srcs:
        o = OBJ / (s.stem + ".o")
        objs.append(o)
        if force or _newer(s, o, headers):
            flags = [f for f in NVCC_FLAGS if f != "--use_fast_math" or s.stem not in EXACT_SOURCES]
            cmd = [nvcc, *flags, "-I", str(kdir), "-c", str(s), "-o", str(o)]
            if verbose:
                cmd.insert(1, "-Xptxas")
                cmd.insert(2, "-v")
            jobs.append(cmd)
    if jobs:
        with cf.ThreadPoolExecutor(max_workers=min(16, len(jobs))) as ex:
            for out in ex.map(_run, jobs):
                if verbose and out.strip():
                    print(out)
    if force or jobs or not KERNEL_LIB.exists():
        _link([nvcc, "-shared", *map(str, objs), "-lcudart"], KERNEL_LIB)
    return KERNEL_LIB


def build_core(force: bool = False) -> Path:
    """Compile the C++ host core (planner, cost model, KV manager, batcher, ...) as a pybind11 module."""
    import pybind11

    srcs = sorted((CSRC / "core").glob("*.cpp")) + sorted((CSRC / "runtime").glob("*.cpp"))
    headers = sorted((CSRC / "core").glob("*.hpp")) + sorted((CSRC / "runtime").glob("*.hpp"))
    if not srcs:
        return core_lib_path()
    inc = ["-I", pybind11.get_include(), "-I", sysconfig.get_paths()["include"], "-I", str(CSRC / "core"),
           "-I", str(CSRC / "runtime")]
    jobs, objs = [], []
    for s in srcs:
        o = OBJ / ("core_" + s.stem + ".o")
        objs.append(o)
        if force or _newer(s, o, headers):
            jobs.append(["g++", *CXX_FLAGS, *inc, "-c", str(s), "-o", str(o)])
    if jobs:
        with cf.ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            list(ex.map(_run, jobs))
    out = core_lib_path()
    if force or jobs or not out.exists():
        _link(["g++", "-shared", *map(str, objs), "-pthread"], out)
    return out


def ensure_built(architecture: str, kernels: bool = True) -> None:
    """What a model of this architecture needs, compiled if it is missing or out of date."""
    with _locked(), cf.ThreadPoolExecutor(max_workers=2) as ex:
        jobs = [ex.submit(build_core)]
        if kernels:
            jobs.append(ex.submit(build_kernels, only=ARCH_SOURCES.get(architecture)))
        for j in jobs:
            j.result()


def build_all(force: bool = False, verbose: bool = False) -> None:
    with _locked():
        build_kernels(force=force, verbose=verbose)
        build_core(force=force)


if __name__ == "__main__":
    build_all(force="--force" in sys.argv, verbose="-v" in sys.argv)
    print("built:", KERNEL_LIB, core_lib_path())
