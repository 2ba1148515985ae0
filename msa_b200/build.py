"""Builds the C-ABI libraries in-tree with nvcc for sm_100a.

    python -m msa_b200.build            # build every library whose sources are newer than it
    python -m msa_b200.build --force

Two libraries, each built only when it is asked for or stale: ``libmsa_b200.so`` (memory routing and sparse attention,
``include/msa_b200.h``) and ``libmsa_b200_lm.so`` (the layered decoder designs, ``include/msa_b200_lm.h``).
"""
from __future__ import annotations

import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libmsa_b200.so")
LIB_LM = os.path.join(HERE, "libmsa_b200_lm.so")
SOURCES = ["cabi.cu", "pool.cu", "bookkeeping.cu", "route_simt.cu", "route_tc.cu", "route_modes.cu", "route_dec.cu", "topk.cu", "gather.cu", "decode_attn.cu", "prefill_attn.cu", "attn_generic.cu", "doc_attn_tc.cu", "decode_dense.cu"]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC"]
LM_SOURCES = ["cabi.cu", "lm_norm.cu", "lm_latent.cu", "lm_attn_tc.cu", "lm_latent_decode.cu", "lm_delta.cu", "lm_delta_chunk.cu", "lm_group.cu", "lm_linear.cu", "lm_linear_chunk.cu", "lm_moe.cu", "lm_moe_tc.cu"]
# name -> (library, sources, extra flags, headers outside csrc).  The decoder designs keep the full accuracy of 32-bit
# divisions, exponentials and angles.
LIBRARIES = {
    "msa": (LIB, SOURCES, ["--use_fast_math"], ["msa_b200.h"]),
    "lm": (LIB_LM, LM_SOURCES, [], ["msa_b200.h", "msa_b200_lm.h"]),
}


def _nvcc() -> str:
    cand = os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "bin", "nvcc")
    return cand if os.path.exists(cand) else "nvcc"


def _stale(name: str) -> bool:
    path, sources, _, headers = LIBRARIES[name]
    if not os.path.exists(path):
        return True
    t = os.path.getmtime(path)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cuh") or f in sources]
    deps += [os.path.join(HERE, "..", "include", h) for h in headers]
    return any(os.path.getmtime(d) > t for d in deps)


def _build_one(name: str, verbose: bool) -> None:
    path, sources, extra, _ = LIBRARIES[name]
    tag = f"{name}.{os.getpid()}"          # two processes may build at once: each its own objects, the library by rename
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)

    def compile_one(src):
        obj = os.path.join(objdir, f"{src[:-3]}.{tag}.o")
        cmd = [_nvcc(), *NVCC_FLAGS, *extra, *os.environ.get("MSA_B200_NVCC_EXTRA", "").split(), "-c", os.path.join(CSRC, src), "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            sys.stderr.write(r.stderr)
        return obj

    with ThreadPoolExecutor(max_workers=min(8, len(sources))) as ex:
        objs = list(ex.map(compile_one, sources))
    part = f"{path}.{os.getpid()}"
    r = subprocess.run([_nvcc(), "-shared", "-o", part, *objs], capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    os.replace(part, path)
    for o in objs:
        os.unlink(o)


def build(force: bool = False, verbose: bool = False, only: str | None = None) -> str:
    """Build what is stale (``only``: one library by name); returns the path of ``only`` or of the routing library."""
    for name in ([only] if only else LIBRARIES):
        if force or _stale(name):
            _build_one(name, verbose)
    return LIBRARIES[only or "msa"][0]


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
