"""Builds the in-tree native libraries.

    python -m trl_b200.csrc.build [--force] [--verbose] [--part layered [--kinds attention,moe]]

* ``trl_b200/_lib/libtrl_b200_kernels.so``  every ``*.cu`` here, compiled by nvcc for sm_100a only
  (``-gencode arch=compute_100a,code=sm_100a``); works without a GPU (cross-compile).
* ``trl_b200/_lib/libtrl_b200_layered.so``  with ``--part layered``: only the sources that serving a layered decoder with
  these mixers and feed-forwards needs, and those of earlier such builds (used when the whole kernel library has not been
  built).
* ``trl_b200/_lib/libtrl_b200_host.so``     ``*.cpp`` host runtime (scheduler, packing), g++ -O3.

Objects are cached next to the sources' hashes, so unchanged files are not recompiled.
"""
from __future__ import annotations

import argparse
import concurrent.futures as cf
import hashlib
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
LIB = os.path.join(os.path.dirname(HERE), "_lib")
OBJ = os.path.join(LIB, "obj")

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "--use_fast_math",
              "-Xcompiler", "-fPIC,-fvisibility=hidden", "-Xptxas", "-v", "--expt-relaxed-constexpr"]
# sources whose results the fast approximations of exp, tanh, erf, division and square root would show in
EXACT_MATH = {"grouped_attn.cu", "hgrn2.cu", "hgrn2_chunk_tcgen05.cu", "layered_moe.cu", "mixers.cu", "mlstm_chunk_tcgen05.cu", "rglru.cu", "rglru_tcgen05.cu"}
# every source here builds into the one library used at any GPU count (no loads shared across a thread-block cluster)


# Parts of the kernel library that can be built alone.  "layered": what every layered decoder needs, and the sources of the
# mixers and feed-forwards it has.
PARTS = {"layered": ("decode.cu", "decode_gemm.cu", "mixers.cu", "tensormap.cu")}
_GROUPED = ("grouped_attn.cu", "grouped_decode_tcgen05.cu", "mixer_attn_tcgen05.cu")
LAYERED_KINDS = {"latent_attention": ("grouped_attn.cu", "latent_decode_tcgen05.cu", "mixer_attn_tcgen05.cu"),
                 "mlstm": ("mlstm_chunk_tcgen05.cu",), "attention": _GROUPED, "attention_2": _GROUPED,
                 "rglru": ("rglru.cu", "rglru_tcgen05.cu"), "hgrn2": ("hgrn2.cu", "hgrn2_chunk_tcgen05.cu"), "moe": ("grouped_gemm_tcgen05.cu", "layered_moe.cu")}


def _nvcc() -> str:
    for c in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if c and os.path.exists(c):
            return c
    raise RuntimeError("nvcc not found")


def _digest(path: str, extra: str) -> str:
    h = hashlib.sha256(extra.encode())
    with open(path, "rb") as f:
        h.update(f.read())
    for hdr in sorted(os.listdir(HERE)):
        if hdr.endswith((".cuh", ".h", ".hpp")):
            with open(os.path.join(HERE, hdr), "rb") as f:
                h.update(f.read())
    return h.hexdigest()[:16]


def _compile(src: str, force: bool, verbose: bool) -> str:
    is_cu = src.endswith(".cu")
    flags = [f for f in NVCC_FLAGS if not (f == "--use_fast_math" and os.path.basename(src) in EXACT_MATH)] if is_cu else ["-O3", "-std=c++17", "-fPIC", "-fvisibility=hidden", "-pthread"]
    tag = _digest(src, " ".join(flags))
    obj = os.path.join(OBJ, f"{os.path.basename(src)}.{tag}.o")
    if os.path.exists(obj) and not force:
        return obj
    for old in os.listdir(OBJ):
        if old.startswith(os.path.basename(src) + "."):
            os.remove(os.path.join(OBJ, old))
    cmd = ([_nvcc()] + flags if is_cu else ["g++"] + flags) + ["-I", HERE, "-c", src, "-o", obj]
    r = subprocess.run(cmd, capture_output=True, text=True)
    log = os.path.join(OBJ, os.path.basename(src) + ".log")
    with open(log, "w") as f:
        f.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
    if verbose or r.returncode != 0:
        sys.stderr.write(r.stdout + r.stderr)
    if r.returncode != 0:
        raise RuntimeError(f"compilation of {src} failed (see {log})")
    return obj


def build(force: bool = False, verbose: bool = False, part: str | None = None, kinds=None) -> dict[str, str]:
    """``kinds`` (with ``part``): the :data:`LAYERED_KINDS` it has to cover, default all of them."""
    os.makedirs(OBJ, exist_ok=True)
    want = set(os.listdir(HERE))
    if part is not None:
        built = {f.split(".cu.")[0] + ".cu" for f in os.listdir(OBJ) if f.endswith(".o")}  # earlier builds' sources stay in
        some = {f for k in (LAYERED_KINDS if kinds is None else kinds) for f in LAYERED_KINDS.get(k, ())}
        every = {f for fs in LAYERED_KINDS.values() for f in fs}
        want &= set(PARTS[part]) | some | (every & built)
    cus = sorted(os.path.join(HERE, f) for f in want if f.endswith(".cu"))
    cpps = sorted(os.path.join(HERE, f) for f in os.listdir(HERE) if f.endswith(".cpp"))
    with cf.ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 2)) as ex:
        cu_objs = list(ex.map(lambda s: _compile(s, force, verbose), cus))
        cpp_objs = list(ex.map(lambda s: _compile(s, force, verbose), cpps))
    out = {}
    if cu_objs:
        so = os.path.join(LIB, f"libtrl_b200_{part or 'kernels'}.so")
        if force or not os.path.exists(so) or any(os.path.getmtime(o) > os.path.getmtime(so) for o in cu_objs):
            cmd = [_nvcc(), "-shared", "-o", so] + cu_objs + ["-gencode", "arch=compute_100a,code=sm_100a",
                                                              "-Xcompiler", "-fPIC", "-cudart", "shared"]
            r = subprocess.run(cmd, capture_output=True, text=True)
            if r.returncode != 0:
                raise RuntimeError("link failed:\n" + r.stdout + r.stderr)
        out["kernels"] = so
    if cpp_objs:
        so = os.path.join(LIB, "libtrl_b200_host.so")
        if force or not os.path.exists(so) or any(os.path.getmtime(o) > os.path.getmtime(so) for o in cpp_objs):
            r = subprocess.run(["g++", "-shared", "-o", so] + cpp_objs + ["-pthread"], capture_output=True, text=True)
            if r.returncode != 0:
                raise RuntimeError("link failed:\n" + r.stdout + r.stderr)
        out["host"] = so
    return out


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    ap.add_argument("--part", choices=sorted(PARTS))
    ap.add_argument("--kinds", help="comma-separated kinds a layered part covers (default: all)")
    a = ap.parse_args()
    for k, v in build(a.force, a.verbose, a.part, a.kinds.split(",") if a.kinds else None).items():
        print(f"{k}: {v}")


if __name__ == "__main__":
    main()
