"""Build recipe for the CUDA libraries: every .cu under csrc/ compiled for sm_100a with nvcc.

Two shared libraries are built in-tree (next to this file), so that they travel with a snapshot of the repository:

    libatma_b200.so     the Polar / gated-delta kernels behind include/atma_b200.h
    libatma_decoder.so  the kernels of the configured decoder models behind include/atma_decoder.h

A translation unit that both need is compiled once and linked into both.  ``build()`` makes both, ``build("decoder")``
only what that library needs.  Nothing else is compiled at run time.
"""

import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
INCLUDE = os.path.join(os.path.dirname(HERE), "include")

LIBS = {"b200": os.path.join(HERE, "libatma_b200.so"), "decoder": os.path.join(HERE, "libatma_decoder.so")}
LIB = LIBS["b200"]

SHARED = {"error.cu", "sm100_host.cu", "decode_linear.cu"}
DECODER = {"decoder_rows.cu", "norm_store.cu", "rotary_store.cu", "softmax_attention.cu", "softmax_prefill_sm100.cu", "softmax_decode_mma.cu",
           "delta_rule.cu", "delta_scan_sm100.cu"}

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr", "-Xptxas", "-v",
]


def sources(which):
    """The translation units of one library."""
    every = {f for f in os.listdir(CSRC) if f.endswith(".cu")}
    return sorted((DECODER | SHARED) & every if which == "decoder" else every - DECODER)


def _stale(target, deps):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def build(which=None, force=False, verbose=False):
    """Compile changed translation units and link.  ``which``: "b200", "decoder" or None for both.  Returns the path of
    the library (of libatma_b200.so when both are built)."""
    nvcc = os.environ.get("NVCC", "nvcc")
    names = list(LIBS) if which is None else [which]
    os.makedirs(OBJ, exist_ok=True)
    headers = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    headers += [os.path.join(INCLUDE, f) for f in os.listdir(INCLUDE) if f.endswith(".h")]
    obj = lambda src: os.path.join(OBJ, src[:-3] + ".o")
    jobs = []
    for src in sorted({s for n in names for s in sources(n)}):
        if force or _stale(obj(src), [os.path.join(CSRC, src)] + headers):
            jobs.append(src)

    def run(cmd, target, what):
        part = f"{target}.{os.getpid()}.part"                  # a concurrent or interrupted build leaves no half file
        r = subprocess.run(cmd + ["-o", part], capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed on {what}:\n{r.stdout}\n{r.stderr}")
        os.replace(part, target)
        return r.stdout + r.stderr

    def compile_one(src):
        report = run([nvcc] + NVCC_FLAGS + ["-x", "cu", "-c", os.path.join(CSRC, src)], obj(src), src)
        with open(obj(src) + ".log", "w") as f:
            f.write(report)
        if verbose:
            print(report)

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        list(ex.map(compile_one, jobs))
    for n in names:
        objs = [obj(s) for s in sources(n)]
        if force or jobs or _stale(LIBS[n], objs):
            run([nvcc, "-shared"] + objs + ["-lcudart"], LIBS[n], os.path.basename(LIBS[n]))
    return LIBS[names[0]]


if __name__ == "__main__":
    only = [a for a in sys.argv[1:] if a in LIBS]
    print(build(only[0] if only else None, force="--force" in sys.argv, verbose="-v" in sys.argv))
