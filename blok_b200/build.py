"""In-tree build of the CUDA library (sm_100a only).

    python -m blok_b200.build            # builds blok_b200/libblok_b200.so and the executables if stale
    python -m blok_b200.build --force
    python -m blok_b200.build --trace-run  # only blok-trace-run, from the sources its models need

nvcc cross-compiles without a GPU.  Objects go to blok_b200/build/, the shared
library next to this file so that it travels with the source tree.
"""
import argparse
import concurrent.futures
import glob
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "libblok_b200.so")
OBJ = os.path.join(HERE, "build")
CLI = os.path.join(HERE, "blok-kimi-exec")
TRACE_RUN = os.path.join(HERE, "blok-trace-run")
# What a model opened from a config.json needs: blok-trace-run is linked from these objects alone.
STACK_SOURCES = ["abi", "batcher", "bf16_kernels", "gemm_f32", "gemm_tma", "grouped_attn", "kv_pages", "latent_attn", "linear_attn", "lm_head",
                 "mla_attend_tc", "model", "model_stack", "nomozen", "pamopel", "prompt_attn_tc", "residual_norm", "residual_streams", "state_space",
                 "table_experts", "wgemm_stream"]

NVCC_FLAGS = [
    "-std=c++17", "-O3", "-lineinfo", "-gencode", "arch=compute_100a,code=sm_100a",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr",
]


# Extra nvcc flags for a one-off build, e.g. BLOK_NVCC_EXTRA="-Xptxas -warn-spills" python -m blok_b200.build --force
EXTRA = os.environ.get("BLOK_NVCC_EXTRA", "").split()


def _deps():
    hdrs = glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(CSRC, "*.h"))
    hdrs.append(os.path.join(HERE, "..", "include", "blok_b200.h"))
    return hdrs


def _compile(src, verbose_ptxas):
    obj = os.path.join(OBJ, os.path.basename(src) + ".o")
    deps = [src] + _deps()
    if os.path.exists(obj) and all(os.path.getmtime(d) <= os.path.getmtime(obj) for d in deps):
        return obj, ""
    cmd = ["nvcc"] + NVCC_FLAGS + EXTRA + (["-Xptxas", "-v"] if verbose_ptxas else []) + ["-c", src, "-o", obj]
    p = subprocess.run(cmd, capture_output=True, text=True)
    if p.returncode != 0:
        raise RuntimeError("nvcc failed for %s:\n%s\n%s" % (src, p.stdout, p.stderr))
    return obj, p.stderr


def _compile_all(srcs, verbose_ptxas=False):
    os.makedirs(OBJ, exist_ok=True)
    with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, len(srcs))) as ex:
        return list(ex.map(lambda s: _compile(s, verbose_ptxas), srcs))


def _stale(out, *deps):
    return not os.path.exists(out) or any(os.path.getmtime(d) > os.path.getmtime(out) for d in deps)


def build_trace_run(force=False):
    """blok-trace-run, compiling only STACK_SOURCES; returns its path."""
    objs = [r[0] for r in _compile_all([os.path.join(CSRC, n + ".cu") for n in STACK_SOURCES])]
    src = os.path.join(HERE, "cli", "blok_trace_run.cpp")
    if force or _stale(TRACE_RUN, src, *objs):
        part = "%s.%d" % (TRACE_RUN, os.getpid())  # moved into place when complete
        subprocess.check_call(["nvcc", "-std=c++17", "-O2", "-gencode", "arch=compute_100a,code=sm_100a", "-I",
                               os.path.join(HERE, "..", "include"), src] + objs + ["-o", part])
        os.replace(part, TRACE_RUN)
    return TRACE_RUN


def build(force=False, verbose_ptxas=False):
    srcs = sorted(glob.glob(os.path.join(CSRC, "*.cu")))
    if force:
        for o in glob.glob(os.path.join(OBJ, "*.o")):
            os.remove(o)
    results = _compile_all(srcs, verbose_ptxas)
    objs = [r[0] for r in results]
    log = "".join(r[1] for r in results)
    if force or not os.path.exists(OUT) or any(os.path.getmtime(o) > os.path.getmtime(OUT) for o in objs):
        cmd = ["nvcc", "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", OUT] + objs + ["-lcudart", "-ldl"]
        subprocess.check_call(cmd)
    cli_src = os.path.join(HERE, "cli", "blok_kimi_exec.cpp")
    if os.path.exists(cli_src) and (force or not os.path.exists(CLI) or os.path.getmtime(cli_src) > os.path.getmtime(CLI)
                                    or os.path.getmtime(OUT) > os.path.getmtime(CLI)):
        subprocess.check_call(["g++", "-std=c++17", "-O2", "-I", os.path.join(HERE, "..", "include"), cli_src, "-o", CLI,
                               "-L", HERE, "-lblok_b200", "-Wl,-rpath,$ORIGIN"])
    build_trace_run(force)
    return OUT, log


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--ptxas", action="store_true", help="print registers / spills / shared memory per kernel")
    ap.add_argument("--trace-run", action="store_true", help="build blok-trace-run only")
    a = ap.parse_args()
    if a.trace_run:
        print(build_trace_run(a.force))
        sys.exit(0)
    out, log = build(a.force, a.ptxas)
    if a.ptxas:
        sys.stderr.write(log)
    print(out)
