"""Builds the sm_100a kernel library in-tree with nvcc (no GPU needed: nvcc cross-compiles).

``python -m tgi_b200.ops.build [SET]`` compiles every ``csrc/*.cu`` with
``-gencode arch=compute_100a,code=sm_100a -lineinfo`` and links ``ops/libtgi_b200_kernels.so``.
The library exposes plain ``extern "C"`` launchers that take raw device pointers and a stream, so it
has no dependency on the PyTorch C++ headers and rebuilds in seconds.

``KERNEL_SETS`` names parts of the library that are enough for some models; such a part becomes a library of its
own, for tools that run one model from a checkout where nothing is built yet.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path
from typing import List, Optional

HERE = Path(__file__).resolve().parent
CSRC = HERE / "csrc"
BUILD_DIR = HERE / "_build"
LIB_PATH = HERE / "libtgi_b200_kernels.so"
KERNEL_SETS = {
    # decoders in bf16 / fp32 on one GPU, with attention, recurrent layers and routed experts
    "decoder": ["attention_prefill_sm100", "attention_sm100", "attn_inputs", "fused_ops", "gemm_sm100", "gemm_static_scratch",
                "latent_attention_sm100", "mixer_ops", "moe_sm100", "recurrent_sm100", "stream_ops"],
}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
    "-diag-suppress", "177",
]


def nvcc_path() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found; set NVCC or install the CUDA toolkit")


def lib_path(kernel_set: Optional[str] = None) -> Path:
    return LIB_PATH if kernel_set is None else HERE / f"libtgi_b200_{kernel_set}.so"


def sources(kernel_set: Optional[str] = None) -> List[Path]:
    if kernel_set is None:
        return sorted(CSRC.glob("*.cu"))
    return [CSRC / f"{name}.cu" for name in KERNEL_SETS[kernel_set]]


def _stale(target: Path, deps: List[Path]) -> bool:
    if not target.exists():
        return True
    t = target.stat().st_mtime
    return any(d.stat().st_mtime > t for d in deps)


def build(force: bool = False, verbose: bool = False, ptxas_info: bool = False, kernel_set: Optional[str] = None) -> Path:
    target = lib_path(kernel_set)
    nvcc = nvcc_path()
    BUILD_DIR.mkdir(exist_ok=True)
    headers = sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h"))
    jobs = []
    objs = []
    for src in sources(kernel_set):
        obj = BUILD_DIR / (src.stem + ".o")
        objs.append(obj)
        if force or _stale(obj, [src] + headers):
            cmd = [nvcc, *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
            if ptxas_info:
                cmd[1:1] = ["-Xptxas", "-v"]
            jobs.append(cmd)

    def run(cmd):
        if verbose:
            print(" ".join(cmd), flush=True)
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed:\n{' '.join(cmd)}\n{r.stdout}\n{r.stderr}")
        if ptxas_info:
            print(r.stderr)

    if jobs:
        with ThreadPoolExecutor(max_workers=min(len(jobs), os.cpu_count() or 4)) as ex:
            list(ex.map(run, jobs))
    if force or jobs or _stale(target, objs):
        run([nvcc, "-shared", "-o", str(target), *map(str, objs), "-lcudart_static", "-ldl", "-lrt", "-lpthread"])
    return target


if __name__ == "__main__":
    named = [a for a in sys.argv[1:] if a in KERNEL_SETS]
    path = build(force="--force" in sys.argv, verbose=True, ptxas_info="--ptxas" in sys.argv,
                 kernel_set=named[0] if named else None)
    print(path)
