"""Builds libironmill_cuda.so (sm_100a only) from csrc/ with nvcc, in-tree.

Run as ``python -m ironmill_b200.build``; also called by ``__graft_entry__.build()``.
nvcc cross-compiles without a GPU, so the library can be built on a CPU-only box and
carried to the B200 machine next to the sources.
"""
from __future__ import annotations

import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "csrc", "_obj")
LIB = os.path.join(HERE, "libironmill_cuda.so")
# A library with one model family only: what a host that serves a single model has to compile.
FAMILY_SOURCES = {
    "stack": ("api.cu", "session.cu", "stack.cu", "dense.cu", "latent_attn.cu", "grouped_attn.cu",
              "linear_attn.cu", "linear_gated.cu"),
}


def family_lib(family: str) -> str:
    return os.path.join(HERE, f"libironmill_cuda_{family}.so")


INCLUDE = os.path.join(os.path.dirname(HERE), "include")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden,-Wall", "--expt-relaxed-constexpr",
]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    return "nvcc"


def _nccl_include() -> list[str]:
    try:
        import nvidia.nccl  # type: ignore

        inc = os.path.join(list(nvidia.nccl.__path__)[0], "include")
        if os.path.exists(os.path.join(inc, "nccl.h")):
            return ["-I", inc]
    except Exception:
        pass
    return []


def sources(family: str | None = None) -> list[str]:
    return sorted(FAMILY_SOURCES[family]) if family else sorted(f for f in os.listdir(CSRC) if f.endswith(".cu"))


def _headers() -> list[str]:
    return [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))] + [os.path.join(INCLUDE, f) for f in os.listdir(INCLUDE)]


def ensure(family: str) -> str:
    """The library a model of `family` runs on: the complete one if it is there and current, else the family's own,
    compiled now if need be."""
    deps = [os.path.join(CSRC, f) for f in sources()] + _headers()
    return LIB if not _stale(LIB, deps) else build(family=family)


def _stale(target: str, deps: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def build(force: bool = False, verbose: bool = False, ptxas_info: bool = False, family: str | None = None) -> str:
    """Compiles what is out of date and links; the complete library, or with `family` that family's."""
    os.makedirs(OBJ, exist_ok=True)
    headers = _headers()
    lib = family_lib(family) if family else LIB
    nvcc = _nvcc()
    jobs = []
    for src in sources(family):
        obj = os.path.join(OBJ, src[:-3] + ".o")
        path = os.path.join(CSRC, src)
        if force or _stale(obj, [path] + headers):
            cmd = [nvcc, *NVCC_FLAGS, *_nccl_include(), "-I", INCLUDE, "-c", path, "-o", obj]
            if ptxas_info:
                cmd[1:1] = ["-Xptxas", "-v"]
            jobs.append((src, cmd))

    def run(job):
        src, cmd = job
        r = subprocess.run(cmd, capture_output=True, text=True)
        return src, r

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        for src, r in ex.map(run, jobs):
            if verbose or ptxas_info or r.returncode != 0:
                sys.stderr.write(f"--- nvcc {src}\n{r.stdout}{r.stderr}")
            if r.returncode != 0:
                raise RuntimeError(f"nvcc failed on {src}")
    objs = [os.path.join(OBJ, s[:-3] + ".o") for s in sources(family)]
    if force or jobs or _stale(lib, objs):
        cmd = [nvcc, "-shared", "-o", lib, *objs, "-lcudart", "-ldl"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
    return lib


if __name__ == "__main__":
    build(force="--force" in sys.argv, verbose="-v" in sys.argv, ptxas_info="--ptxas" in sys.argv)
    print(LIB)
