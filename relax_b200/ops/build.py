"""In-tree build of the sm_100a extension.

Kernels live in ``csrc/*.cu`` and do not include PyTorch headers (nvcc compiles
each in seconds); ``csrc/bindings*.cpp`` adapt tensors to the C launchers.  The
result is ``relax_b200/_C.so`` beside the Python sources, so it travels with the
tree to a GPU machine and is the file the ops import.
"""
from __future__ import annotations

import os
import subprocess
import sys
import sysconfig
from concurrent.futures import ThreadPoolExecutor

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
CSRC = os.path.join(ROOT, "csrc")
OBJ = os.path.join(ROOT, "build", "obj")
SO_PATH = os.path.join(ROOT, "relax_b200", "_C.so")
# The serving extension: the kernels and bindings a composed stack's engine launches, and nothing else.  It is built where
# only such an engine runs and the full extension has not been built (a fresh checkout); the ops load whichever exists.
SERVING_SO_PATH = os.path.join(ROOT, "relax_b200", "_C_serving.so")
SERVING_SOURCES = ["attention_fwd_sm100.cu", "decode_attn_tc_sm100.cu", "decode_step_sm100.cu", "gemm2_sm100.cu", "gemm_decode_sm100.cu", "gemm_sm100.cu",
                   "gqa_stack_sm100.cu", "head_gemm_sm100.cu", "hgrn2_chunk_sm100.cu", "latent_attn_sm100.cu", "mingru_sm100.cu", "moe_gemm_sm100.cu",
                   "moe_stack_sm100.cu", "paged_flash_sm100.cu", "stack_sm100.cu", "stream_sm100.cu", "talk_decode_sm100.cu", "talk_flash_sm100.cu",
                   "bindings_serving.cpp", "launch_count.cpp", "module_serving.cpp"]
# fp32 results of these kernels are compared at fp32 rounding: IEEE division, square root and library exponentials
PRECISE_SOURCES = {"stack_sm100.cu", "gqa_stack_sm100.cu", "mingru_sm100.cu", "moe_stack_sm100.cu", "stream_sm100.cu"}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "--use_fast_math",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr", "-Xptxas", "-v",
]


def _nvcc() -> str:
    cand = os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "bin", "nvcc")
    return cand if os.path.exists(cand) else "nvcc"


def _stale(out: str, deps: list) -> bool:
    if not os.path.exists(out):
        return True
    t = os.path.getmtime(out)
    return any(os.path.getmtime(d) > t for d in deps)


def _run(cmd: list, log_path: str | None = None):
    p = subprocess.run(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if log_path:
        with open(log_path, "w") as f:
            f.write(" ".join(cmd) + "\n" + p.stdout)
    if p.returncode != 0:
        raise RuntimeError(f"command failed: {' '.join(cmd)}\n{p.stdout[-6000:]}")
    return p.stdout


def ensure_serving(verbose: bool = False) -> str:
    """The extension a serving process needs: the full one when it is there and newer than the sources, else the serving
    subset (built if missing or stale).  Concurrent callers take turns."""
    import fcntl

    srcs = [os.path.join(CSRC, f) for f in os.listdir(CSRC)]
    if not _stale(SO_PATH, srcs):
        return SO_PATH
    os.makedirs(OBJ, exist_ok=True)
    with open(os.path.join(OBJ, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return build_extension(verbose, serving=True)


def build_extension(verbose: bool = False, force: bool = False, serving: bool = False) -> str:
    """Compile what is stale and link the full extension, or (``serving``) the serving subset."""
    import torch
    from torch.utils import cpp_extension as ce

    os.makedirs(OBJ, exist_ok=True)
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".h", ".cuh"))]
    names = SERVING_SOURCES if serving else [f for f in os.listdir(CSRC) if f != "module_serving.cpp"]
    so_path = SERVING_SO_PATH if serving else SO_PATH
    cus = sorted(f for f in names if f.endswith(".cu"))
    cpps = sorted(f for f in names if f.endswith(".cpp"))
    jobs = []
    objs = []
    for f in cus:
        src, out = os.path.join(CSRC, f), os.path.join(OBJ, f + ".o")
        objs.append(out)
        if force or _stale(out, [src] + headers):
            flags = [x for x in NVCC_FLAGS if not (f in PRECISE_SOURCES and x == "--use_fast_math")]
            jobs.append(([_nvcc()] + flags + ["-I", CSRC, "-c", src, "-o", out], out + ".log"))
    abi = int(getattr(torch._C, "_GLIBCXX_USE_CXX11_ABI", True))
    inc = []
    for p in ce.include_paths("cuda") if "device_type" in ce.include_paths.__code__.co_varnames else ce.include_paths(True):
        inc += ["-isystem", p]
    inc += ["-isystem", sysconfig.get_paths()["include"], "-I", CSRC]
    cxx = os.environ.get("CXX", "g++")
    for f in cpps:
        src, out = os.path.join(CSRC, f), os.path.join(OBJ, f + ".o")
        objs.append(out)
        if force or _stale(out, [src] + headers):
            jobs.append(([cxx, "-O2", "-std=c++17", "-fPIC", f"-D_GLIBCXX_USE_CXX11_ABI={abi}",
                          "-DTORCH_EXTENSION_NAME=_C", "-DTORCH_API_INCLUDE_EXTENSION_H", "-w"] + inc +
                         ["-c", src, "-o", out], out + ".log"))
    if jobs:
        if verbose:
            print(f"[relax_b200.build] compiling {len(jobs)} translation unit(s) for sm_100a", flush=True)
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            list(ex.map(lambda j: _run(*j), sorted(jobs, key=lambda j: -os.path.getsize(j[0][j[0].index("-c") + 1]))))
    if jobs or force or _stale(so_path, objs):
        tlib = os.path.join(os.path.dirname(torch.__file__), "lib")
        cuda_lib = os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "lib64")
        cmd = [cxx, "-shared", "-o", so_path] + objs + [
            f"-L{tlib}", "-lc10", "-ltorch", "-ltorch_cpu", "-ltorch_python", "-lc10_cuda", "-ltorch_cuda",
            f"-L{cuda_lib}", "-lcudart", f"-Wl,-rpath,{tlib}", f"-Wl,-rpath,{cuda_lib}",
        ]
        _run(cmd)
        if verbose:
            print(f"[relax_b200.build] linked {so_path}", flush=True)
    return so_path


def ptxas_report() -> str:
    """Concatenated ``-Xptxas -v`` output of the last build (registers, spills, shared memory)."""
    out = []
    for f in sorted(os.listdir(OBJ)) if os.path.isdir(OBJ) else []:
        if f.endswith(".cu.o.log"):
            out.append(open(os.path.join(OBJ, f)).read())
    return "\n".join(out)


if __name__ == "__main__":
    build_extension(verbose=True, force="--force" in sys.argv)
