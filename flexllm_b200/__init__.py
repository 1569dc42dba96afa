"""flexllm_b200 -- B200 (sm_100a) kernels for FlexLLM's quantized Llama-3.2-1B operator path and the models built on
the same runner.

The product is ``libflexllm_b200.so`` (CUDA kernels behind the C ABI of ``include/flexllm_b200.h``)
plus the C++ host API in ``include/flexllm/``. This Python package is plumbing only: it loads the
library with ctypes and hands it host buffers (``models``: registry, configuration, generation; no torch needed) or
device pointers of torch tensors (``ops``, whose names are also available here). There is no CPU or PyTorch
fallback: if the library is missing or a call fails, an exception is raised.
"""
import importlib

from . import _lib


def __getattr__(name):          # the operators (and with them torch) are imported when first asked for
    if name.startswith("__"):
        raise AttributeError(name)
    ops = importlib.import_module(".ops", __name__)
    return ops if name == "ops" else getattr(ops, name)
