"""Builds the CUDA library of this package in-tree for sm_100a.

    python cccc-lite_b200/build.py            # build if sources are newer than the library
    python cccc-lite_b200/build.py --force

Three libraries, in the order of their dependence:
  libcccc-b200-decoder.so   layer operations of decoders with BF16 / float weights (csrc/decoder/, see
                            include/cccc_b200_decoder.h) and the serving core: model registry, KV cache, scheduler,
                            generation loop, the models made of these operations (csrc/host/)
  libcccc-cuda-b200.so      the drop-in for the reference's `cccc-cuda` plug-in library on the quantized-weight linear
                            path (csrc/*.cu, see include/cccc_cuda_b200.h)
  libcccc-b200-host.so      the quantized models and the reference's Matrix / Cublas interface, on top of both
A process that serves a model of the first library needs no other: build_decoder() compiles just that one.
"""
from __future__ import annotations

import glob
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libcccc-cuda-b200.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")

FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "--extended-lambda",
    "-Xcompiler", "-fPIC,-fvisibility=hidden", "-shared", "-cudart", "shared",
]


def sources() -> list[str]:
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")))


def stale() -> bool:
    if not os.path.exists(LIB):
        return True
    t = os.path.getmtime(LIB)
    deps = sources() + glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(HERE, "..", "include", "*.h"))
    return any(os.path.getmtime(d) > t for d in deps)


HOST_LIB = os.path.join(HERE, "libcccc-b200-host.so")
HOST_DIR = os.path.join(CSRC, "host")
DECODER_LIB = os.path.join(HERE, "libcccc-b200-decoder.so")
DECODER_DIR = os.path.join(CSRC, "decoder")
OBJ_DIR = os.path.join(HERE, "build")    # git-ignored object files: only changed translation units are recompiled
# the serving core; every other .cpp of csrc/host belongs to the host library
CORE = ["gpu_control", "json", "tensor_source", "kv_cache", "language_model", "generate", "scheduler", "layered_decoder", "layered_mixers", "design_config",
        "fakilorn", "tazunex", "model_capi"]


def _mtime(paths) -> float:
    return max(os.path.getmtime(p) for p in paths)


def _headers() -> list[str]:
    return glob.glob(os.path.join(HERE, "..", "include", "*.h"))


def _run_all(jobs) -> None:
    from concurrent.futures import ThreadPoolExecutor

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as pool:
        for cmd, rc in zip(jobs, pool.map(subprocess.call, jobs)):
            if rc != 0:
                raise subprocess.CalledProcessError(rc, cmd[0])


class _Lock:
    """One build at a time in a checkout."""

    def __enter__(self):
        import fcntl

        os.makedirs(OBJ_DIR, exist_ok=True)
        self.f = open(os.path.join(OBJ_DIR, ".lock"), "w")
        fcntl.flock(self.f, fcntl.LOCK_EX)

    def __exit__(self, *_):
        self.f.close()


def build_decoder(force: bool = False, verbose: bool = False) -> str:
    """Compiles and links libcccc-b200-decoder.so, only what is stale."""
    cuda = os.path.dirname(os.path.dirname(NVCC))
    cu = sorted(glob.glob(os.path.join(DECODER_DIR, "*.cu")))
    cpp = [os.path.join(HOST_DIR, n + ".cpp") for n in CORE]
    cu_deps = _mtime(glob.glob(os.path.join(DECODER_DIR, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.cuh")) + _headers())
    cpp_deps = _mtime(glob.glob(os.path.join(HOST_DIR, "*.h")) + _headers())
    with _Lock():
        jobs, objs = [], []
        for src in cu + cpp:
            is_cu = src.endswith(".cu")
            obj = os.path.join(OBJ_DIR, ("decoder_" if is_cu else "core_") + os.path.splitext(os.path.basename(src))[0] + ".o")
            objs.append(obj)
            if force or not os.path.exists(obj) or os.path.getmtime(obj) < max(os.path.getmtime(src), cu_deps if is_cu else cpp_deps):
                if is_cu:
                    jobs.append([NVCC] + [f for f in FLAGS if f != "-shared"] + (["-Xptxas", "-v"] if verbose else []) + ["-c", "-o", obj, src])
                else:
                    jobs.append(["g++", "-std=c++17", "-O2", "-fPIC", "-pthread", f"-I{cuda}/include", "-c", "-o", obj, src])
        _run_all(jobs)
        if jobs or not os.path.exists(DECODER_LIB) or os.path.getmtime(DECODER_LIB) < _mtime(objs):
            subprocess.check_call([NVCC, "-shared", "-cudart", "shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", DECODER_LIB + ".new"] + objs)
            os.replace(DECODER_LIB + ".new", DECODER_LIB)
    return DECODER_LIB


def host_stale() -> bool:
    if not os.path.exists(HOST_LIB):
        return True
    t = os.path.getmtime(HOST_LIB)
    deps = glob.glob(os.path.join(HOST_DIR, "*")) + glob.glob(os.path.join(HERE, "..", "include", "*.h")) + [LIB, DECODER_LIB]
    return any(os.path.getmtime(d) > t for d in deps)


def build_host(force: bool = False) -> str:
    """The C++ host layer (Matrix / Cublas / GpuControl mirror) on top of the CUDA library."""
    if force or host_stale():
        cuda = os.path.dirname(os.path.dirname(NVCC))
        cmd = ["g++", "-std=c++17", "-O2", "-fPIC", "-pthread", "-shared", "-fvisibility=hidden", f"-I{cuda}/include", "-o", HOST_LIB]
        cmd += [s for s in sorted(glob.glob(os.path.join(HOST_DIR, "*.cpp"))) if os.path.splitext(os.path.basename(s))[0] not in CORE]
        cmd += [f"-L{HERE}", "-lcccc-cuda-b200", "-lcccc-b200-decoder", f"-L{cuda}/lib64", "-lcublas", "-lcudart", "-Wl,-rpath,$ORIGIN"]
        subprocess.check_call(cmd)
    return HOST_LIB


def _object_stale(src: str, obj: str) -> bool:
    if not os.path.exists(obj):
        return True
    t = os.path.getmtime(obj)
    deps = [src] + glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(HERE, "..", "include", "*.h"))
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False) -> str:
    """Compiles every translation unit of csrc/ for sm_100a (in parallel, only the stale ones) and links the library."""
    build_decoder(force, verbose)
    if force or stale():
        os.makedirs(OBJ_DIR, exist_ok=True)
        compile_flags = [f for f in FLAGS if f != "-shared"]
        extra = os.environ.get("B200_NVCC_EXTRA", "").split()
        jobs = []
        for src in sources():
            obj = os.path.join(OBJ_DIR, os.path.basename(src)[:-3] + ".o")
            if force or extra or _object_stale(src, obj):
                jobs.append([NVCC] + compile_flags + extra + (["-Xptxas", "-v"] if verbose else []) + ["-c", "-o", obj, src])
        _run_all(jobs)
        objs = [os.path.join(OBJ_DIR, os.path.basename(src)[:-3] + ".o") for src in sources()]
        subprocess.check_call([NVCC, "-shared", "-cudart", "shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", LIB] + objs)
    build_host(force)
    return LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
