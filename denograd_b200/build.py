"""Builds libjsgrad_cuda.so (hand-written sm_100a kernels + the C ABI) in-tree with nvcc."""
from __future__ import annotations

import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT_DIR = os.path.join(HERE, "lib")
LIB = os.path.join(OUT_DIR, "libjsgrad_cuda.so")
# The whole library is every source below.  A component is the part one model family needs on its own, linked as a
# library of that name, so that a fresh checkout which serves one model does not compile the other families' kernels.
CORE = ["device.cu", "comm.cu", "elementwise.cu", "sample.cu", "tensor_map.cu"]
DENSE, RECURRENT, BRANCHES = ["dense.cu", "dense_tc.cu"], ["recurrent.cu", "latent_attn.cu"], ["linear_state.cu", "window_attn.cu"]
COMPONENTS = {"hybrid": CORE + DENSE + RECURRENT + BRANCHES, "hybrid_recurrent": CORE + DENSE + RECURRENT, "hybrid_branches": CORE + DENSE + BRANCHES}
# which of them a mixer of the layer-list models is in
MIXER_COMPONENT = {"mingru": "hybrid_recurrent", "delta": "hybrid_recurrent", "latent_attention": "hybrid_recurrent", "mlstm": "hybrid_branches",
                   "parallel": "hybrid_branches", "window_attention": "hybrid_branches", "lightning": "hybrid_branches"}
SOURCES = CORE + ["gemv.cu", "matvec_w8.cu", "gemm_small.cu", "gemm_tc.cu", "attention.cu", "attention_chunk.cu", "step.cu", "program.cu",
                  *DENSE, *RECURRENT, *BRANCHES]
ARCH = ["-gencode", "arch=compute_100a,code=sm_100a"]
FLAGS = ["-O3", "-std=c++17", "-lineinfo", "-Xcompiler", "-fPIC,-fvisibility=hidden", "--expt-relaxed-constexpr"]


def component_of(mixers) -> str:
    """The smallest component with the kernels of these kinds of mixer."""
    names = {MIXER_COMPONENT.get(m, "hybrid") for m in mixers}
    return names.pop() if len(names) == 1 else "hybrid"


def nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _headers() -> list[str]:
    return [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))] + [os.path.join(HERE, "..", "include", "jsgrad_cuda.h")]


def fresh(component: str | None = None) -> bool:
    """Whether the library (of a component, or the whole one) exists and is newer than everything it is made of."""
    lib = os.path.join(OUT_DIR, f"libjsgrad_cuda_{component}.so") if component else LIB
    return not _stale(lib, [os.path.join(CSRC, f) for f in (COMPONENTS[component] if component else SOURCES)] + _headers())


def build(force: bool = False, verbose: bool = False, component: str | None = None) -> str:
    os.makedirs(OUT_DIR, exist_ok=True)
    lib = os.path.join(OUT_DIR, f"libjsgrad_cuda_{component}.so") if component else LIB
    headers = _headers()
    objs = []
    procs = []
    for src in COMPONENTS[component] if component else SOURCES:
        s = os.path.join(CSRC, src)
        o = os.path.join(OUT_DIR, src.replace(".cu", ".o"))
        objs.append(o)
        if force or _stale(o, [s] + headers):
            cmd = [nvcc(), *ARCH, *FLAGS, "-c", s, "-o", o]
            if verbose:
                cmd.insert(1, "-Xptxas=-v")
            procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0 or verbose:
            sys.stderr.write(f"--- {src}\n{out}\n")
        failed |= p.returncode != 0
    if failed:
        raise RuntimeError("nvcc failed")
    if force or procs or _stale(lib, objs):
        part = f"{lib}.{os.getpid()}"
        subprocess.run([nvcc(), *ARCH, "-shared", "-o", part, *objs, "-Xcompiler", "-fPIC", "-ldl"], check=True)
        os.replace(part, lib)
    return lib


if __name__ == "__main__":
    names = [a for a in sys.argv[1:] if a in COMPONENTS]
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv, component=names[0] if names else None))
