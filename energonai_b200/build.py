"""Builds libenergon_b200.so (the C-ABI CUDA library) in-tree with nvcc for sm_100a.

    python -m energonai_b200.build [--force] [--verbose]

Every .cu under csrc/ is compiled to an object under build/ (skipped when up to date) and
linked into energonai_b200/libenergon_b200.so.  No torch headers are involved.
"""
import concurrent.futures
import fcntl
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ_DIR = os.path.join(os.path.dirname(HERE), "build", "energon_b200")
LIB_PATH = os.path.join(HERE, "libenergon_b200.so")

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "--use_fast_math", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
              "-diag-suppress", "177,550"]
# Recurrences add up the logarithms of their gates over a whole sequence: an approximation's bias would
# add up with them, so these files get the accurate functions; so do angles that grow with the position.
ACCURATE = {"matrix_memory.cu", "matrix_memory_tc.cu", "decay_memory.cu", "decay_memory_tc.cu", "attention_rotary.cu", "latent_inputs.cu",
            "selective_scan.cu"}


def nvcc_flags(source):
    return [f for f in NVCC_FLAGS if not (f == "--use_fast_math" and source in ACCURATE)]


def _nvcc():
    cand = os.path.join(os.environ.get("CUDA_HOME", "/usr/local/cuda"), "bin", "nvcc")
    return cand if os.path.exists(cand) else "nvcc"


def _newer(src_paths, target):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(p) > t for p in src_paths)


def build(force=False, verbose=False):
    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(OBJ_DIR, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)          # processes that start together build once
        return _build(force, verbose)


def _build(force, verbose):
    sources = sorted(f for f in os.listdir(CSRC) if f.endswith(".cu"))
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h", ".inc"))]
    headers.append(os.path.join(os.path.dirname(HERE), "include", "energon_b200.h"))
    jobs = []
    for s in sources:
        src, obj = os.path.join(CSRC, s), os.path.join(OBJ_DIR, s[:-3] + ".o")
        if force or _newer([src] + headers, obj):
            jobs.append([_nvcc()] + nvcc_flags(s) + (["-Xptxas", "-v"] if verbose else []) + ["-c", src, "-o", obj])

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        return cmd, r

    with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        for cmd, r in ex.map(run, jobs):
            if verbose or r.returncode != 0:
                sys.stderr.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
            if r.returncode != 0:
                raise RuntimeError(f"nvcc failed for {cmd[-3]}")
    objs = [os.path.join(OBJ_DIR, s[:-3] + ".o") for s in sources]
    if force or jobs or _newer(objs, LIB_PATH):
        cmd = [_nvcc(), "-shared", "-o", LIB_PATH] + objs + ["-gencode", "arch=compute_100a,code=sm_100a"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link of libenergon_b200.so failed")
    return LIB_PATH


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
