"""Builds libbpdq.so in-tree with nvcc for sm_100a.  No JIT cache, no torch extension
machinery: the shared library is plain C ABI and is loaded with ctypes."""
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libbpdq.so")
SOURCES = ["runtime.cu", "dequant_q4k.cu", "gemv_q4k.cu", "gemv_batch.cu", "gemv_persistent.cu", "gemv_stream.cu", "q8_0.cu", "w4a32.cu", "decode_ops.cu", "gemm_q4k_mma.cu", "gemm_q4k_tc5.cu", "gemm_q4k_rg16.cu", "gemm_q8_0_tiles.cu", "llama_forward.cu", "peer_exchange.cu",
           "linear.cu", "decayed_scan.cu", "latent_attention.cu", "delta_rule.cu", "grouped_attention.cu", "residual_streams.cu", "hybrid_forward.cu"]
# The sources some model families need: a process that only serves one of those (bin/trace_run in a fresh checkout)
# compiles and loads these as a library of their own when the whole one has not been built.
PARTS = {"hybrid": ["runtime.cu", "decode_ops.cu", "linear.cu", "decayed_scan.cu", "latent_attention.cu", "delta_rule.cu", "grouped_attention.cu",
                    "residual_streams.cu", "hybrid_forward.cu"]}
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr",
]


def _nvcc():
    for cand in (shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found: libbpdq.so cannot be built")


def lib_path(part=None):
    return LIB if part is None else os.path.join(HERE, f"libbpdq_{part}.so")


def _stale(lib):
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC)]
    deps.append(os.path.join(HERE, "..", "include", "bpdq.h"))
    return any(os.path.getmtime(d) > t for d in deps)


def build(force=False, verbose=False, part=None):
    """Compile every .cu (of a part) to an object, in parallel, and link libbpdq.so (libbpdq_<part>.so)."""
    lib = lib_path(part)
    if not force and not _stale(lib):
        return lib
    nvcc = _nvcc()
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    procs = []
    for src in SOURCES if part is None else PARTS[part]:
        obj = os.path.join(objdir, src.replace(".cu", ".o"))
        cmd = [nvcc, *NVCC_FLAGS, *os.environ.get("BPDQ_NVCC_FLAGS", "").split(), "-c", os.path.join(CSRC, src), "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        procs.append((src, obj, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    objs = []
    for src, obj, p in procs:
        out, _ = p.communicate()
        if verbose or p.returncode:
            sys.stderr.write(out)
        if p.returncode:
            raise RuntimeError(f"nvcc failed on {src}")
        objs.append(obj)
    tmp = f"{lib}.{os.getpid()}"
    subprocess.check_call([nvcc, "-shared", "-o", tmp, *objs, "-gencode", "arch=compute_100a,code=sm_100a"])
    os.replace(tmp, lib)
    return lib


if __name__ == "__main__":
    build(force=True, verbose="-v" in sys.argv)
    print(LIB)
