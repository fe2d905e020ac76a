"""Python face of ``csrc/dyntanh.cu``: the sum into the residual stream and the norm without statistics behind it."""
from __future__ import annotations

from typing import Optional

import torch

from ._lib import KernelError, c_float, c_int, check, check_bias, dt_code, fn, ptr, require_cuda, stream


def add_dyn_tanh(h: torch.Tensor, delta: Optional[torch.Tensor], alpha: float, gain: torch.Tensor, shift: torch.Tensor,
                 out_dtype: torch.dtype, *, delta_bias: Optional[torch.Tensor] = None,
                 rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``h += delta + delta_bias`` (float32 ``h [T, width]``; nothing is added without ``delta``; written back unless
    ``rows`` is given), then ``tanh(alpha h) * gain + shift`` in ``out_dtype``, of all rows or of ``rows`` (int32) only."""
    require_cuda(h, delta, gain, shift, delta_bias, rows)
    T, W = h.shape
    if h.dtype != torch.float32 or any(t.dtype != torch.float32 or t.numel() != W for t in (gain, shift)):
        raise KernelError(f"the residual stream, gain and shift are float32, one element per column ({W})")
    check_bias(delta_bias, W)
    if delta is not None and delta.shape != h.shape:
        raise KernelError("delta must have the residual stream's shape")
    R = T if rows is None else rows.numel()
    out = torch.empty((R, W), dtype=out_dtype, device=h.device)
    check(fn("dyntanh", "sx_add_dyn_tanh")(
        ptr(h), ptr(delta), c_int(dt_code(delta.dtype) if delta is not None else 0), ptr(delta_bias), c_float(alpha), ptr(gain),
        ptr(shift), ptr(out), c_int(dt_code(out_dtype)), ptr(rows), c_int(R), c_int(W), c_int(1 if rows is None else 0), stream()),
        "add_dyn_tanh")
    return out
