"""Build libcera_cuda.so (sm_100a) from cera_b200/csrc with nvcc.

The library is built in-tree so that it travels with the source tree; nothing
is JIT-compiled at import time.  Run it by path, `python cera_b200/build.py [--force] [-v]`:
importing the package itself requires the library to exist already.
"""
import concurrent.futures
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ_DIR = os.path.join(HERE, "_obj")
LIB = os.path.join(HERE, "libcera_cuda.so")

# The library's parts: a build may take only what a model needs (bin/trace_run in a fresh checkout); the default is all.
# Everything that is not listed belongs to "quantized".
PARTS = {"core": ["runtime.cu", "model.cu", "argmax.cu"],
         "layered": ["layered.cu", "dense.cu", "dense_gemv.cu", "dense_gemm.cu", "dense_gemm_tc.cu", "mingru.cu", "latent_attention.cu",
                     "attention_tc.cu", "grouped_attention.cu", "conv.cu", "rglru.cu", "ssm.cu", "ssm_chunk.cu",
                     "moe_route.cu"]}
ALL_PARTS = ("core", "layered", "quantized")
# Translation units whose float arithmetic must not be contracted into FMAs.
NO_FMAD = {"convert.cu"}

ARCH = ["-gencode", "arch=compute_100a,code=sm_100a"]
COMMON = ["-O3", "-std=c++17", "-lineinfo", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
          "--expt-relaxed-constexpr"]


def nvcc():
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found: the CUDA library cannot be built")
    return exe


def _headers():
    hs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    hs.append(os.path.join(os.path.dirname(HERE), "include", "cera_cuda.h"))
    return hs


def _stale(target, deps):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _sources(parts):
    listed = [f for p in PARTS.values() for f in p]
    rest = [f for f in sorted(os.listdir(CSRC)) if f.endswith(".cu") and f not in listed]
    # moe_route.cu is shared: part of either build
    return [f for p in parts for f in (rest + ["moe_route.cu"] if p == "quantized" else PARTS[p])]


def build(force=False, verbose=False, parts=ALL_PARTS):
    os.makedirs(OBJ_DIR, exist_ok=True)
    hdrs = _headers()
    jobs = []
    objs = []
    for src in dict.fromkeys(_sources(parts)):
        s = os.path.join(CSRC, src)
        o = os.path.join(OBJ_DIR, src.replace(".cu", ".o"))
        objs.append(o)
        if force or _stale(o, [s] + hdrs):
            cmd = [nvcc()] + ARCH + COMMON + (["-fmad=false"] if src in NO_FMAD else [])
            if verbose:
                cmd += ["-Xptxas", "-v"]
            cmd += ["-c", s, "-o", o]
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        return cmd, r

    if jobs:
        with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            for cmd, r in ex.map(run, jobs):
                if verbose or r.returncode:
                    sys.stderr.write(" ".join(cmd[-3:]) + "\n" + r.stdout + r.stderr)
                if r.returncode:
                    raise RuntimeError("nvcc failed for " + cmd[-3])
    made_of = os.path.join(OBJ_DIR, "linked.txt")  # the objects the library was linked from
    before = open(made_of).read().split() if os.path.exists(made_of) else []
    if jobs or force or _stale(LIB, objs) or before != [os.path.basename(o) for o in objs]:
        cmd = [nvcc()] + ARCH + ["-shared", "-o", LIB] + objs
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
        with open(made_of, "w") as f:
            f.write("\n".join(os.path.basename(o) for o in objs))
    return LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
