"""Builds mongoose_b200/libmongoose_kernels.so with nvcc for sm_100a only.

The counterpart of the reference's kernel provisioning
(kernel_provision.go:28-88): one shared library with plain C symbols that the
host side opens with dlopen.  Unlike the reference it never probes the GPU for
an architecture (the target is fixed) and never installs a toolkit.

    python -m mongoose_b200.build [--force] [--verbose] [--family=layered]
"""
from __future__ import annotations

import glob
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
INCLUDE = os.path.join(os.path.dirname(HERE), "include")
LIB_NAME = "libmongoose_kernels.so"
LIB_PATH = os.path.join(HERE, LIB_NAME)
# translation unit -> what it serves: "abi" the reference's C symbols, "core" the engine's host code,
# "dense" the fixed seven-matrix decode block, "layered" models described layer by layer
UNITS = {
    "engine.cu": "core",
    "legacy_ops.cu": "abi", "block_ops.cu": "abi",
    "layered_decode.cu": "layered", "layered_prefill.cu": "layered", "gemm_tc.cu": "layered", "gate_attn_tc.cu": "layered",
    "latent_attn.cu": "layered", "latent_attn_tc.cu": "layered", "wkv.cu": "layered", "moe.cu": "layered",
    "dense_phases.cu": "dense", "mega_single.cu": "dense", "mega_tp.cu": "dense",
}
# A family of models can be served by a library of its own, compiled from what that family needs (the
# persistent kernel of the dense family alone takes two minutes); the whole library serves every family.
FAMILIES = {"layered": ("core", "layered")}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC,-fvisibility=hidden,-ffp-contract=off",
    "--expt-relaxed-constexpr",
    "-Xptxas", "-v",
] + (["-DMK_PROBE_P=" + os.environ["MK_PROBE_P"]] if os.environ.get("MK_PROBE_P") else [])


def _nvcc() -> str:
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(nvcc):
        raise RuntimeError("nvcc not found: the CUDA toolkit is required to build " + LIB_NAME)
    return nvcc


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def family_lib(family: str) -> str:
    """Path of the library that serves one family only."""
    return os.path.join(HERE, f"libmongoose_{family}.so")


def headers() -> list[str]:
    return sorted(glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h")) +
                  [os.path.join(INCLUDE, "mongoose_kernels.h"), os.path.abspath(__file__)])


def fresh(lib: str) -> bool:
    """Is `lib` newer than every source it may have been built from?"""
    return not _stale(lib, [os.path.join(CSRC, u) for u in UNITS] + headers())


def ensure(family: str) -> str:
    """A library that serves `family`: the whole one where it is up to date, else the family's own,
    compiled if need be."""
    return LIB_PATH if fresh(LIB_PATH) else build(family=family)


def build(force: bool = False, verbose: bool = False, family: str | None = None) -> str:
    nvcc = _nvcc()
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    common = headers()
    parts = FAMILIES[family] if family else None
    sources = [u for u, part in UNITS.items() if parts is None or part in parts]
    lib_path = family_lib(family) if family else LIB_PATH
    jobs = []
    objs = []
    for src in sources:
        s = os.path.join(CSRC, src)
        o = os.path.join(objdir, src.replace(".cu", ".o"))
        objs.append(o)
        if force or _stale(o, [s] + common):
            jobs.append((s, o))

    def compile_one(job):
        s, o = job
        cmd = [nvcc, *NVCC_FLAGS, "-c", s, "-o", o]
        r = subprocess.run(cmd, capture_output=True, text=True)
        log = os.path.splitext(o)[0] + ".ptxas.log"
        with open(log, "w") as f:
            f.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {s}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            sys.stderr.write(r.stderr)

    with ThreadPoolExecutor(max_workers=len(sources)) as ex:
        list(ex.map(compile_one, jobs))

    if force or jobs or _stale(lib_path, objs):
        part = f"{lib_path}.{os.getpid()}"
        cmd = [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", part, *objs,
               "-Xcompiler", "-fPIC", "-cudart", "static"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
        os.replace(part, lib_path)
    return lib_path


if __name__ == "__main__":
    p = build(force="--force" in sys.argv, verbose="--verbose" in sys.argv,
              family=next((a.split("=", 1)[1] for a in sys.argv if a.startswith("--family=")), None))
    print(p)
