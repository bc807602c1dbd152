"""Builds libferrum_cuda.so in-tree with nvcc for sm_100a (cross-compiles without a GPU).

    python -m ferrum_cpu_b200.build [--verbose]

A component is a library of its own with the sources one model family needs, for a host that serves
only that family and has nothing built yet: `ensure(component)` returns the complete library when it is
up to date, else builds the component (objects are shared with the complete build).
"""
import concurrent.futures
import contextlib
import fcntl
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB = os.path.join(HERE, "libferrum_cuda.so")
# what every decoder of a model folder needs, and what each design adds
FOLDER = ["common.cu", "codec.cpp", "model_dir.cpp", "decoder.cu", "gemm_bf16.cu", "gemv_bf16.cu", "flash_tc.cu", "flash_f32.cu", "llama_ops.cu", "sample.cu"]
NURINEX = ["mix_rows.cu", "talk_attn.cu", "wkv.cu", "mixer_decode.cu", "nurinex.cu"]
ZOGEVIK = ["post_norm_rows.cu", "rot_attn.cu", "attn_decode.cu", "experts.cu", "zogevik.cu"]
SOURCES = ["gguf_load.cpp", "gemv.cu", "gemv_stream.cu", "rowops.cu", "attn.cu", "gemm_simt.cu", "gemm_tc.cu", "attn_tc.cu",
           "decode_mega.cu", "decode_batch.cu", "llama.cu", "rowq.cu", "ggml_linear.cu", "api.cu"] + FOLDER + NURINEX + ZOGEVIK
COMPONENTS = {"nurinex": FOLDER + NURINEX, "zogevik": FOLDER + ZOGEVIK}
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-Wall",
]


def component_lib(component):
    return os.path.join(HERE, f"libferrum_cuda_{component}.so")


def _nvcc():
    return shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"


def _newer(target, deps):
    if not os.path.exists(target):
        return False
    t = os.path.getmtime(target)
    return all(os.path.getmtime(d) <= t for d in deps)


def _deps(src):
    deps = [os.path.join(CSRC, src)] + [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    deps.append(os.path.join(HERE, "..", "include", "ferrum_cuda.h"))
    return deps


def _compile(src, verbose):
    obj = os.path.join(OBJ, src + ".o")
    if _newer(obj, _deps(src)):
        return obj, ""
    cmd = [_nvcc(), *NVCC_FLAGS, "-x", "cu", "-c", os.path.join(CSRC, src), "-o", obj]
    if verbose:
        cmd[1:1] = ["-Xptxas", "-v"]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"nvcc failed on {src}:\n{r.stdout}\n{r.stderr}")
    return obj, r.stderr


@contextlib.contextmanager
def _lock():
    os.makedirs(OBJ, exist_ok=True)
    with open(os.path.join(OBJ, ".lock"), "w") as f:
        fcntl.flock(f, fcntl.LOCK_EX)
        yield


def build(verbose=False, component=None):
    sources, lib = (SOURCES, LIB) if component is None else (COMPONENTS[component], component_lib(component))
    with _lock():
        with concurrent.futures.ThreadPoolExecutor(max_workers=8) as ex:
            results = list(ex.map(lambda s: _compile(s, verbose), sources))
        objs = [o for o, _ in results]
        log = "".join(l for _, l in results)
        if not _newer(lib, objs):
            part = f"{lib}.{os.getpid()}"
            r = subprocess.run([_nvcc(), "-shared", "-o", part, *objs, "-cudart", "static"], capture_output=True, text=True)
            if r.returncode != 0:
                raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
            os.replace(part, lib)
    return log


def ensure(component):
    """Path of a library that holds the component: the complete one when it is newer than every source, else the
    component's own, compiled now if need be."""
    if _newer(LIB, {d for s in SOURCES for d in _deps(s)}):
        return LIB
    build(component=component)
    return component_lib(component)


if __name__ == "__main__":
    out = build(verbose="--verbose" in sys.argv)
    if out:
        print(out)
    print(LIB)
