"""Builds libpace_b200.so (sm_100a) in-tree with nvcc.

    python amd-pace_b200/build.py [--force] [--verbose]

The shared library exports the C ABI declared in include/pace_b200.h; the Python
package loads it with ctypes.  nvcc cross-compiles without a GPU.
"""
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "pace_b200", "libpace_b200.so")
SOURCES = ["kv_pool.cu", "attn_decode.cu", "attn_mma.cu", "attn_api.cu", "linear_skinny.cu",
           "hybrid_ops.cu", "attn_general.cu", "recurrent.cu", "lightning.cu", "attn_span.cu", "attn_span_keys.cu", "attn_span_umma.cu", "latent.cu", "moe.cu",
           "conv_append.cu", "ssd.cu", "ssd_chunk.cu", "delta.cu", "delta_chunk.cu", "rotate_append.cu", "shift_norm.cu", "attn_pooled.cu",
           "attn_pooled_umma.cu", "gla.cu", "gla_chunk.cu"]
# fp32 exp, log and divide of these files are the accurate ones (they serve 32-bit models)
PRECISE = {"hybrid_ops.cu", "attn_general.cu", "recurrent.cu", "lightning.cu", "latent.cu", "moe.cu", "conv_append.cu",
           "ssd.cu", "ssd_chunk.cu", "delta.cu", "delta_chunk.cu", "rotate_append.cu", "shift_norm.cu", "attn_pooled.cu", "gla.cu",
           "gla_chunk.cu"}
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
         "--use_fast_math", "-Xcompiler", "-fPIC", "-I", os.path.join(ROOT, "include"), "-I", CSRC] + \
    os.environ.get("PACE_NVCC_EXTRA", "").split()


def _newer(a, b):
    return not os.path.exists(b) or os.path.getmtime(a) > os.path.getmtime(b)


def build(force=False, verbose=False):
    srcs = [os.path.join(CSRC, s) for s in SOURCES if os.path.exists(os.path.join(CSRC, s))]
    # every source includes the public header and may include any of the .cuh files
    headers = sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith(".cuh"))
    headers.append(os.path.join(ROOT, "include", "pace_b200.h"))
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    objs, procs = [], []
    for s in srcs:
        o = os.path.join(objdir, os.path.basename(s) + ".o")
        objs.append(o)
        if force or any(_newer(d, o) for d in [s] + headers):
            flags = [f for f in FLAGS if f != "--use_fast_math" or os.path.basename(s) not in PRECISE]
            cmd = [NVCC] + flags + (["-Xptxas", "-v"] if verbose else []) + ["-c", s, "-o", o]
            procs.append((s, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    failed = False
    for s, pr in procs:
        out, _ = pr.communicate()
        if pr.returncode != 0 or verbose:
            print(f"--- {os.path.basename(s)}\n{out}")
        failed |= pr.returncode != 0
    if failed:
        raise RuntimeError("nvcc failed")
    if force or procs or not os.path.exists(OUT):
        subprocess.check_call([NVCC, "-shared", "-o", OUT] + objs + ["-lcudart"])
    return OUT


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
