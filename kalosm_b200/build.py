"""Builds libfusor_b200.so (hand-written CUDA for sm_100a + the C ABI) in-tree with nvcc."""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libfusor_b200.so")
SOURCES = ["api.cu", "repack.cu", "qgemv.cu", "qgemv1.cu", "q5gemv.cu", "dense.cu", "dense_tc.cu", "qgemm.cu", "ops.cu", "attention.cu", "attn_prefill.cu", "attn_prefill_tc.cu", "attn_decode_tc.cu",
           "fused_step.cu", "llama.cu", "hybrid.cu", "delta_rule.cu", "latent_attn.cu", "latent_prefill.cu", "group_attn.cu", "linear_attn.cu", "linear_prefill.cu", "comm.cu", "sampling.cu"]
HEADERS = ["common.cuh", "formats.cuh", "qgemv_common.cuh", "qgemv1_groups.cuh", "packed_act.cuh",
           "attn_decode.cuh", "attn_mma.cuh", "qgemv1_groups2.cuh", "fused_step.cuh", "decoder.cuh", "dense.cuh", "mixers.cuh", "state_columns.cuh", "tcgen05.cuh", os.path.join("..", "..", "include", "fusor_b200.h")]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden", "--expt-relaxed-constexpr"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", shutil.which("nvcc")):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found; libfusor_b200.so cannot be built")


# What a decoder of token-mixer layers over dense weights needs. A library of this part alone has the other sources'
# functions as stubs that answer FB200_ERR_UNSUPPORTED_DTYPE, and lacks their C entry points.
DENSE_PART = ["api.cu", "repack.cu", "dense.cu", "dense_tc.cu", "ops.cu", "sampling.cu", "llama.cu", "hybrid.cu", "delta_rule.cu",
              "latent_attn.cu", "latent_prefill.cu", "group_attn.cu", "linear_attn.cu", "linear_prefill.cu"]
DENSE_LIB = os.path.join(HERE, "libfusor_b200_dense.so")


def _hash(names) -> str:
    h = hashlib.sha256()
    for name in names:
        with open(os.path.join(CSRC, name), "rb") as f:
            h.update(f.read())
    h.update(" ".join(NVCC_FLAGS).encode())
    return h.hexdigest()


def _current(path: str, stamp: str) -> bool:
    if not os.path.exists(path) or not os.path.exists(path + ".stamp"):
        return False
    with open(path + ".stamp") as f:
        return f.read().strip() == stamp


def _mark(path: str, stamp: str) -> None:
    with open(path + ".stamp", "w") as f:
        f.write(stamp)


def _stub_object(objs, objdir: str) -> str:
    """An object that defines the library-internal functions `objs` use but do not define."""
    defined, used = set(), set()
    for line in subprocess.run(["nm", "--no-sort"] + objs, capture_output=True, text=True, check=True).stdout.splitlines():
        parts = line.split()
        if len(parts) >= 2 and "fb200_" in parts[-1]:
            (used if parts[-2] == "U" else defined).add(parts[-1])
    src = os.path.join(objdir, "stubs.c")
    with open(src, "w") as f:
        for name in sorted(used - defined):
            f.write(f"__attribute__((visibility(\"hidden\"))) int {name}(void) {{ return -2; }}\n")
    obj = src[:-2] + ".o"
    subprocess.run(["gcc", "-O1", "-fPIC", "-c", src, "-o", obj], check=True)
    return obj


def build(force: bool = False, verbose: bool = False, part: str = "all") -> str:
    """Compiles the sources that changed for sm_100a and links the shared library; returns its path. part "dense"
    builds only what dense token-mixer decoders need (or returns the whole library if that is current)."""
    whole = _hash(SOURCES + HEADERS)
    if not force and _current(LIB, whole):
        return LIB
    sources, lib = (SOURCES, LIB) if part == "all" else (DENSE_PART, DENSE_LIB)
    stamp = whole if part == "all" else _hash(sources + HEADERS)
    if not force and _current(lib, stamp):
        return lib
    nvcc = _nvcc()
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    procs, objs = [], []
    for src in sources:
        obj = os.path.join(objdir, src.replace(".cu", ".o"))
        objs.append(obj)
        key = _hash([src] + HEADERS)
        if not force and not verbose and _current(obj, key):
            continue
        cmd = [nvcc] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + \
              ["-c", os.path.join(CSRC, src), "-o", obj]
        procs.append((obj, key, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT)))
    failed = False
    for obj, key, p in procs:
        out, _ = p.communicate()
        if verbose or p.returncode:
            sys.stderr.write(out.decode())
        failed |= p.returncode != 0
        if not p.returncode:
            _mark(obj, key)
    if failed:
        raise RuntimeError("nvcc failed")
    link = objs if part == "all" else objs + [_stub_object(objs, objdir)]
    subprocess.run([nvcc, "-shared", "-o", lib] + link + ["-gencode", "arch=compute_100a,code=sm_100a"],
                   check=True)
    _mark(lib, stamp)
    return lib


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
