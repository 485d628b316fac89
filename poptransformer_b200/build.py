"""Builds libpt_b200.so in-tree with nvcc for sm_100a (cross-compiles without a GPU)."""
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.environ.get("PT_B200_LIB", os.path.join(HERE, "libpt_b200.so"))   # same override as _lib.LIB_PATH
SOURCES = ["api.cu", "linear.cu", "attention.cu", "ops.cu", "decode_llama.cu", "decode_llama_short.cu", "gemm_tc.cu", "prefill.cu",
           "gemm_f32.cu", "hyper.cu", "window_attn.cu", "ssm.cu", "post_norm.cu", "moe.cu", "mlstm.cu", "latent.cu", "shift_norm.cu"]
# Sources of a library that serves one architecture: what a program builds that runs only that model and finds no full library.
_SEQUENCES = ["api.cu", "ops.cu", "linear.cu", "gemm_tc.cu", "gemm_f32.cu", "window_attn.cu"]
PARTS = {"Sabisun": _SEQUENCES + ["hyper.cu", "ssm.cu"], "Padetar": _SEQUENCES + ["post_norm.cu", "moe.cu", "mlstm.cu"],
         "Pivavik": _SEQUENCES + ["post_norm.cu", "moe.cu", "latent.cu"], "Puputar": _SEQUENCES + ["shift_norm.cu", "moe.cu", "latent.cu"]}
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "--threads", "0",
    "-Xcompiler", "-fPIC", "-shared",
]


def part_path(part):
    return LIB[:-3] + "_" + part.lower() + ".so"


def needs_build(lib=None):
    lib = lib or LIB
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC)] + [os.path.join(HERE, "..", "include", "pt_b200.h")]
    return any(os.path.getmtime(d) > t for d in deps)


def build_for(architecture):
    """A library that has the kernels of `architecture`: the full one if it is there and current, else one with that part only."""
    if architecture not in PARTS or not needs_build():
        return build()
    return build(part=architecture)


def build(force=False, verbose=False, part=None):
    lib = part_path(part) if part else LIB
    if not force and not needs_build(lib):
        return lib
    tmp = f"{lib[:-3]}.{os.getpid()}.tmp.so"                 # renamed when complete: nobody loads half a library
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    extra = os.environ.get("PT_NVCC_EXTRA", "").split()      # e.g. -DPT_MK_TRACE_WAITS for a diagnostics build
    cmd = [nvcc] + NVCC_FLAGS + extra + (["-Xptxas", "-v"] if verbose else []) + [os.path.join(CSRC, s) for s in (PARTS[part] if part else SOURCES)] + ["-o", tmp]
    res = subprocess.run(cmd, capture_output=True, text=True)
    if verbose or res.returncode != 0:
        sys.stderr.write(res.stdout + res.stderr)
    if res.returncode != 0:
        raise RuntimeError(f"nvcc failed building {os.path.basename(lib)}")
    os.replace(tmp, lib)
    return lib


if __name__ == "__main__":
    build(force=True, verbose=True)
    print(LIB)
