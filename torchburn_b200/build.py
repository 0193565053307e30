"""Builds libtorchburn_b200.so (sm_100a) from csrc/ with nvcc.

    python -m torchburn_b200.build [--force] [--verbose] [--profile full|dense]

The library is written in-tree (torchburn_b200/lib/); it is the only compute
path of the package - nothing falls back to the CPU when it is missing.

Profile "full" (the default) is the whole library.  Profile "dense" leaves the
INT4 kernels out (its INT4 entry points answer TB_ERR_UNSUPPORTED) and is what a
layered model needs; ``ensure`` builds it only where no full library is at hand.
"""
from __future__ import annotations

import concurrent.futures as cf
import fcntl
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "lib", "obj")
LIB = os.path.join(HERE, "lib", "libtorchburn_b200.so")
PROFILES = {"full": LIB, "dense": os.path.join(HERE, "lib", "libtorchburn_b200_dense.so")}
INT4_SOURCES = ("w4_step.cu", "w4_stream.cu", "w4_gemv.cu", "w4_mma.cu", "w4_tc5.cu", "attention.cu")
INT4_ABSENT = "w4_absent.cpp"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden,-Wall", "--expt-relaxed-constexpr",
]


def _nvcc() -> str:
    for cand in (os.environ.get("TB_NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found: the sm_100a library cannot be built")


def sources(profile: str = "full"):
    drop = (INT4_ABSENT,) if profile == "full" else INT4_SOURCES
    return sorted(f for f in os.listdir(CSRC) if f.endswith((".cu", ".cpp")) and f not in drop)


def _newest_header() -> float:
    hdrs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    hdrs.append(os.path.join(HERE, "..", "include", "torchburn_b200.h"))
    return max(os.path.getmtime(h) for h in hdrs)


def up_to_date(profile: str = "full") -> bool:
    lib = PROFILES[profile]
    if not os.path.exists(lib):
        return False
    newest = max(_newest_header(), *(os.path.getmtime(os.path.join(CSRC, f)) for f in sources(profile)))
    return os.path.getmtime(lib) >= newest


def ensure(profile: str) -> str:
    """The library a model of this profile runs on: the full one if it is built, else the profile's own,
    compiled now if need be."""
    if up_to_date("full"):
        return PROFILES["full"]
    return PROFILES[profile] if up_to_date(profile) else build(profile=profile)


def build(force: bool = False, verbose: bool = False, profile: str = "full") -> str:
    os.makedirs(OBJ, exist_ok=True)
    with open(os.path.join(HERE, "lib", ".lock"), "w") as lock:   # two processes of a fresh checkout
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build(force, verbose, profile)


def _build(force: bool, verbose: bool, profile: str) -> str:
    LIB = PROFILES[profile]
    nvcc = _nvcc()
    hdr_time = _newest_header()
    jobs = []
    objs = []
    for src in sources(profile):
        sp = os.path.join(CSRC, src)
        op = os.path.join(OBJ, os.path.splitext(src)[0] + ".o")
        objs.append(op)
        if force or not os.path.exists(op) or os.path.getmtime(op) < max(os.path.getmtime(sp), hdr_time):
            cmd = [nvcc, *NVCC_FLAGS, "-x", "cu", "-c", sp, "-o", op]
            if verbose:
                cmd.insert(1, "-Xptxas=-v")
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("nvcc failed:\n" + " ".join(cmd) + "\n" + r.stdout + r.stderr)
        return r.stderr

    if jobs:
        with cf.ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            for out in ex.map(run, jobs):
                if verbose and out:
                    print(out)
    if jobs or force or not os.path.exists(LIB):
        # -fvisibility=hidden + explicit export of the extern "C" API keeps the symbol table to the ABI
        tmp = LIB + ".tmp"
        link = [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", tmp, *objs,
                "-Xlinker", "--no-undefined", "-ldl", "-lpthread"]
        run(link)
        os.replace(tmp, LIB)  # atomic: a reader never sees a half-written library
    return LIB


if __name__ == "__main__":
    prof = sys.argv[sys.argv.index("--profile") + 1] if "--profile" in sys.argv else "full"
    path = build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, profile=prof)
    print(path)
