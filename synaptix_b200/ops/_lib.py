"""Calling the compiled kernels: pointers, dtype codes, streams, error codes."""
from __future__ import annotations

import contextlib
import ctypes
from typing import Optional

import torch

from ..csrc.build import KernelsUnavailable, load_library
from .options import OPTIONS as _PDL_OPTION

_DT = {torch.float32: 0, torch.bfloat16: 1}

_ERRORS = {10001: "unsupported dtype combination", 10002: "unsupported size", 10003: "misaligned pointer or stride",
           10004: "a bounded wait inside the kernel ran out (see the kernel's status word)",
           10005: "the problem needs more scratch than the library's built-in array holds"}


class KernelError(RuntimeError):
    """A kernel refused its arguments or its launch failed."""


def dt_code(dtype: torch.dtype) -> int:
    try:
        return _DT[dtype]
    except KeyError:
        raise KernelError(f"kernels take float32 and bfloat16 tensors, not {dtype}") from None


def require_cuda(*tensors: Optional[torch.Tensor]) -> None:
    for t in tensors:
        if t is None:
            continue
        if not t.is_cuda:
            raise KernelsUnavailable(
                "this operation runs only as a CUDA kernel on an sm_100a device; it was given a "
                f"{t.device} tensor (there is no CPU path)")
        if not t.is_contiguous():
            raise KernelError("kernels take contiguous tensors")


def ptr(t: Optional[torch.Tensor]) -> ctypes.c_void_p:
    return ctypes.c_void_p(0 if t is None else t.data_ptr())


try:                                    # the raw handle without building a Stream object (an order of magnitude cheaper)
    _raw_stream = torch._C._cuda_getCurrentRawStream
except AttributeError:                  # pragma: no cover - older torch
    _raw_stream = None


def stream() -> ctypes.c_void_p:
    """The current CUDA stream of the current device (the capturing stream inside a graph capture)."""
    if _raw_stream is not None:
        return ctypes.c_void_p(_raw_stream(torch.cuda.current_device()))
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


def check_bias(bias: Optional[torch.Tensor], n: int) -> None:
    if bias is not None and (bias.dtype != torch.float32 or bias.numel() != n):
        raise KernelError(f"a product's bias is float32 with one element per output ({n})")


def check_resid_tanh(x, w, bias, h, gain, shift) -> None:
    """What the products that end in the residual stream and its norm without statistics have in common."""
    (M, K), (N, K2) = x.shape, w.shape
    if K != K2 or tuple(h.shape) != (M, N) or h.dtype != torch.float32:
        raise KernelError("the residual stream must be contiguous float32 [M, N]")
    check_bias(bias, N)
    if any(t.dtype != torch.float32 or t.numel() != N for t in (gain, shift)):
        raise KernelError("gain and shift of the norm are float32 [N]")


_COUNTER = [None]


def set_launch_counter(obj) -> None:
    """``obj.kernel_launches`` is incremented for every kernel launched from here on."""
    _COUNTER[0] = obj


def count_launches(n: int) -> None:
    if _COUNTER[0] is not None:
        _COUNTER[0].kernel_launches += n


def check(code: int, what: str, launches: int = 1) -> None:
    if code == 0:
        if _COUNTER[0] is not None:
            _COUNTER[0].kernel_launches += launches
        return
    if code in _ERRORS:
        raise KernelError(f"{what}: {_ERRORS[code]}")
    raise KernelError(f"{what}: CUDA error {code} at launch")


_FN_CACHE = {}
_LIBS = {}


def _library(lib: str):
    """The loaded library; the launch options of this process are handed to it when it is loaded."""
    h = _LIBS.get(lib)
    if h is None:
        h = _LIBS[lib] = load_library(lib)
        _set_pdl(lib)
    return h


def loaded(lib: str) -> bool:
    return lib in _LIBS


# Whether kernels are launched with programmatic dependent launch: the option of that name, and off inside
# ``late_launch``.  A library is told when one of its functions is next asked for.
_LATE = [0]
_LIB_PDL = {}


def _want_pdl() -> bool:
    return bool(_PDL_OPTION.pdl) and not _LATE[0]


def _set_pdl(lib: str) -> None:
    want = _want_pdl()
    f = getattr(_LIBS[lib], "sx_set_pdl", None)
    if f is not None:
        f(ctypes.c_int(1 if want else 0))
    _LIB_PDL[lib] = want


def apply_pdl() -> None:
    """Tell every loaded library whether kernels are launched with programmatic dependent launch."""
    for lib in _LIBS:
        _set_pdl(lib)


@contextlib.contextmanager
def late_launch(on: bool = True):
    """Kernels launched inside are scheduled when the kernel before them has ended, not while it runs.  For a kernel whose
    blocks would otherwise hold the SMs' shared memory and registers, waiting, while another branch's kernel that could
    run looks for room (blocks that run beside each other on two streams)."""
    if not on:
        yield
        return
    _LATE[0] += 1
    try:
        yield
    finally:
        _LATE[0] -= 1


def fn(lib: str, name: str):
    key = (lib, name)
    f = _FN_CACHE.get(key)
    if f is None:
        f = getattr(_library(lib), name)
        f.restype = ctypes.c_int
        _FN_CACHE[key] = f
    if _LIB_PDL[lib] is not (not _LATE[0] and _PDL_OPTION.pdl):
        _set_pdl(lib)
    return f


c_int = ctypes.c_int
c_float = ctypes.c_float
c_longlong = ctypes.c_longlong
c_ulonglong = ctypes.c_ulonglong


# ---------------------------------------------------------------------------------------------------------------
# The gated activation of the products' "silu_mul" epilogue.  (0, 0) is silu(g) * u; (alpha, limit) with limit > 0 is
# g' sigmoid(alpha g') (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit); ``form="gelu_tanh"`` is
# gelu_tanh(g) * u (the tanh form of GELU; alpha and limit unused).  A feed-forward that wants another form than the
# first runs its gate/up product inside ``gate_activation(...)``; the faces of the products call ``use_gate`` before a
# launch with that epilogue, which tells the library if its last value was another one.  ``form="relu2"`` is for the
# experts' products of ONE matrix (``moe_up``): relu(z)^2.
# ---------------------------------------------------------------------------------------------------------------
GATE_FORMS = {"sigmoid": 0, "gelu_tanh": 1, "relu2": 2}
_GATE = [(0.0, 0.0, 0)]
_LIB_GATE = {}


@contextlib.contextmanager
def gate_activation(alpha: float = 0.0, limit: float = 0.0, form: str = "sigmoid"):
    old = _GATE[0]
    _GATE[0] = (float(alpha), float(limit), GATE_FORMS[form])
    try:
        yield
    finally:
        _GATE[0] = old


def current_gate():
    """``(alpha, limit, form code)`` of the gated activation in force."""
    return _GATE[0]


def use_gate(lib: str) -> None:
    want = _GATE[0]
    if _LIB_GATE.get(lib) != want:
        f = getattr(_library(lib), "sx_set_gate_act")
        f.restype = None
        f(ctypes.c_float(want[0]), ctypes.c_float(want[1]), ctypes.c_int(want[2]))
        _LIB_GATE[lib] = want
