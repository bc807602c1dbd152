"""Which class serves which architecture, and `load`: a path in, a model on a GPU out.

A folder (config.json + model.safetensors) names its architecture in the configuration; a file is a GGUF,
whose header says gpt2, llama or qwen2.
"""
import os

from . import _lib
from ._lib import FerrumCudaError

DTYPES = {"float32": _lib.FC_MATH_FP32, "bfloat16": _lib.FC_MATH_BF16}
F32_MODES = (_lib.FC_MATH_FP32, _lib.FC_MATH_BF16X3)


def _folder(name):
    """Loader of the design with that class in decoder.py."""
    def load_folder(path, device, math_mode, ctx):
        from . import decoder
        return getattr(decoder, name)(path, device=device, math_mode=_lib.FC_MATH_BF16 if math_mode is None else math_mode,
                                      ctx=ctx or decoder.DEFAULT_CTX)
    return load_folder


def _gguf_mode(math_mode):
    mode = _lib.FC_MATH_FP32 if math_mode is None else math_mode
    if mode not in F32_MODES:
        raise FerrumCudaError(_lib.FC_E_ARG, "Q8_0 models run in f32 arithmetic (FC_MATH_FP32 or FC_MATH_BF16X3)")
    return mode


def _gpt2(path, device, math_mode, ctx):
    from .engine import CudaSlm
    return CudaSlm.from_gguf(path, device=device, math_mode=_gguf_mode(math_mode))


def _llama(path, device, math_mode, ctx):
    from .llama import CudaLlama
    return CudaLlama.from_gguf(path, device=device, math_mode=_gguf_mode(math_mode), ctx_cap=ctx or 0)


# architecture -> (loader, component of the library that holds its kernels; None: the complete library)
ARCHITECTURES = {
    "gpt2": (_gpt2, None),
    "llama": (_llama, None),
    "qwen2": (_llama, None),
    "Nurinex": (_folder("CudaNurinex"), "nurinex"),
    "Zogevik": (_folder("CudaZogevik"), "zogevik"),
}


def architecture(path):
    if os.path.isdir(path):
        from .decoder import dir_architecture
        return dir_architecture(path)
    from . import engine, llama
    try:
        engine.gguf_probe(path)
        return "gpt2"
    except FerrumCudaError:
        llama.gguf_probe(path)
        return "llama"                          # the same class serves qwen2 files


def load(path, device=0, math_mode=None, ctx=0):
    """The model at `path` on a GPU. math_mode None: the architecture's default; ctx 0: its default context."""
    arch = architecture(path)
    if arch not in ARCHITECTURES:
        raise FerrumCudaError(_lib.FC_E_FORMAT, f"no model class serves the architecture {arch!r}")
    return ARCHITECTURES[arch][0](path, device, math_mode, ctx)
