"""The loaded library and the error type, without torch."""
import ctypes as C

from . import _lib

_handle = None


class FlexLLMError(RuntimeError):
    def __init__(self, fn, status):
        l = lib()
        msg = l.flexllm_status_string(status).decode()
        super().__init__(f"{fn} failed: {msg} (status {status}, cuda error {l.flexllm_last_cuda_error()})")
        self.status = status


def lib():
    global _handle
    if _handle is None:
        _handle = _lib.load()
    return _handle


def check(fn, st):
    if st != 0:
        raise FlexLLMError(fn, st)


def call(name, *args):
    """A library call on host buffers (default stream)."""
    check(name, getattr(lib(), name)(*args))
