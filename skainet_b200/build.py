"""Builds libskainet_cuda.so in-tree with nvcc for sm_100a (cross-compiles without a GPU).

    python -m skainet_b200.build [--force] [--verbose]

`build` makes the whole library; `build_family` compiles only what one model family runs (FAMILIES), for a
program that serves a single model from a fresh checkout.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libskainet_cuda.so")
OBJ_DIR = os.path.join(HERE, "build")

ARCH = ["-gencode", "arch=compute_100a,code=sm_100a"]
COMMON = ["-O3", "-std=c++17", "-lineinfo", "-Xcompiler", "-fPIC,-Wall,-Wno-unused-function",
          "-I", os.path.join(ROOT, "include"), "-I", CSRC]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


# translation units of a model family (the entry points of the others are absent from its library)
DENSE = ["skn_core.cu", "skn_kv_cache.cu", "skn_dense.cu", "skn_rows.cu", "skn_mixers.cu", "skn_glue.cu", "skn_decoder.cu"]
FAMILIES = {"lugasun": DENSE + ["skn_lugasun.cu"],
            "tutezen": DENSE + ["skn_ssm.cu", "skn_latent.cu", "skn_moe.cu", "skn_tutezen.cu"]}


def sources(family: str | None = None) -> list[str]:
    return sorted(os.path.join(CSRC, f) for f in (FAMILIES[family] if family else os.listdir(CSRC)) if f.endswith(".cu"))


def _deps_mtime(family: str | None = None) -> float:
    files = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if not f.endswith(".cu")] + sources(family)
    return max(os.path.getmtime(f) for f in files + [os.path.join(ROOT, "include", "skainet_cuda.h")])


def _fresh(lib: str, family: str | None = None) -> bool:
    return os.path.exists(lib) and os.path.getmtime(lib) >= _deps_mtime(family)


def build_family(family: str) -> str:
    """Path of a library with this family's entry points: the whole library when it is built, else a smaller one."""
    return LIB if _fresh(LIB) else _build(os.path.join(HERE, f"libskainet_{family}.so"), family)


def build(force: bool = False, verbose: bool = False) -> str:
    return _build(LIB, None, force, verbose)


def _build(LIB: str, family: str | None, force: bool = False, verbose: bool = False) -> str:
    if not force and _fresh(LIB, family):
        return LIB
    nvcc = _nvcc()
    os.makedirs(OBJ_DIR, exist_ok=True)
    hdr_mtime = max(os.path.getmtime(os.path.join(CSRC, f)) for f in os.listdir(CSRC) if not f.endswith(".cu"))
    hdr_mtime = max(hdr_mtime, os.path.getmtime(os.path.join(ROOT, "include", "skainet_cuda.h")))
    objs, procs = [], []
    for src in sources(family):
        obj = os.path.join(OBJ_DIR, os.path.basename(src)[:-3] + ".o")
        objs.append(obj)
        if not force and os.path.exists(obj) and os.path.getmtime(obj) >= max(os.path.getmtime(src), hdr_mtime):
            continue
        cmd = [nvcc, *ARCH, *COMMON, "-c", src, "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas")
            cmd.insert(2, "-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        if p.returncode != 0:
            failed = True
            sys.stderr.write(f"nvcc failed on {src}:\n{out}\n")
        elif verbose or out.strip():
            sys.stderr.write(out)
    if failed:
        raise RuntimeError("nvcc compilation failed")
    link = [nvcc, *ARCH, "-shared", "-o", LIB, *objs, "-cudart", "static"]
    r = subprocess.run(link, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if r.returncode != 0:
        raise RuntimeError("link failed:\n" + r.stdout)
    return LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
