"""Python faces of the kernels in ``csrc/parallel.cu``: the sum of a layer's scaled branches into the residual stream,
fused with one or two RMS norms of the same row, and a scale of float32 rows in place."""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ._lib import KernelError, c_float, c_int, c_longlong, check, dt_code, fn, ptr, require_cuda, stream


def _weighted(terms: Sequence):
    """A second term that is a mixture's unformed weighted sum (``WeightedRows``, without a factor of its own): the terms
    with its rows in its place, and ``(place, weights)``; else the terms as they are and ``None``."""
    from .normed import WeightedRows
    terms = [(x.materialize() if isinstance(x, WeightedRows) and i != 1 else x, s) for i, (x, s) in enumerate(terms)]
    if len(terms) == 2 and isinstance(terms[1][0], WeightedRows):
        wr = terms[1][0]
        if wr.rows.dtype != torch.float32:
            raise KernelError("the rows of a weighted sum are float32")
        return terms[:1], (wr, terms[1][1])
    return terms, None


def _terms(h: torch.Tensor, terms: Sequence):
    terms = [(x.materialize() if hasattr(x, "materialize") else x, s) for x, s in terms]
    if len(terms) > 2:
        raise KernelError("at most two scaled terms are added in one pass")
    out = []
    for x, s in terms:
        require_cuda(x, s)
        if x.shape != h.shape:
            raise KernelError("a term must have the residual stream's shape")
        if s is not None and (s.dtype != torch.float32 or s.numel() != h.shape[1]):
            raise KernelError("a term's factor is a float32 vector over the width")
        out.append((x, s))
    while len(out) < 2:
        out.append((None, None))
    return out


def add_scaled_rmsnorm(h: torch.Tensor, terms: Sequence, gains: Sequence[Optional[torch.Tensor]], eps: float,
                       out_dtype: torch.dtype, rows: Optional[torch.Tensor] = None) -> List[torch.Tensor]:
    """``h += sum_i s_i * x_i`` (``terms``: up to two ``(x_i [T, width], s_i float32 [width] or None)``; written back
    unless ``rows`` is given), then one RMS norm per entry of ``gains`` (one or two float32 vectors) of the same rows:
    ``rmsnorm(h) * gain`` in ``out_dtype``, for all rows or for ``rows`` (int32) only.  A single gain of ``None``: the
    rows of the stream themselves in ``out_dtype``.  The second term may be a ``WeightedRows``, formed on the way."""
    require_cuda(h, rows, *gains)
    if len(gains) == 2 and None in gains:
        raise KernelError("rows without a norm stand alone")
    if h.dtype != torch.float32 or any(g is not None and (g.dtype != torch.float32 or g.numel() != h.shape[1]) for g in gains):
        raise KernelError("the residual stream and norm gains are float32, one gain per column")
    if not 1 <= len(gains) <= 2:
        raise KernelError("one or two norms")
    terms, weighted = _weighted(terms)
    (a, sa), (b, sb) = _terms(h, terms)
    place = wts = None
    top = 0
    if weighted is not None:
        wr, sb = weighted
        if tuple(wr.shape) != tuple(h.shape) or (sb is not None and (sb.dtype != torch.float32 or sb.numel() != h.shape[1])):
            raise KernelError("a term must have the residual stream's shape")
        b, place, wts, top = wr.rows, wr.place, wr.weights, wr.weights.shape[1]
        require_cuda(b, place, wts, sb)
    T, H = h.shape
    R = T if rows is None else rows.numel()
    ys = [torch.empty((R, H), dtype=out_dtype, device=h.device) for _ in gains]
    check(fn("parallel", "sx_add_scaled_rmsnorm")(
        ptr(h), ptr(a), c_int(dt_code(a.dtype) if a is not None else 0), ptr(sa),
        ptr(b), c_int(dt_code(b.dtype) if b is not None else 0), ptr(sb), ptr(gains[0]),
        ptr(gains[1] if len(gains) > 1 else None), c_float(eps), ptr(ys[0]), ptr(ys[1] if len(ys) > 1 else None), ptr(rows),
        c_int(R), c_int(H), c_int(dt_code(out_dtype)), c_int(1 if rows is None else 0), ptr(place), ptr(wts), c_int(top), stream()),
        "add_scaled_rmsnorm")
    return ys


def add_scaled(h: torch.Tensor, terms: Sequence) -> None:
    """``h += sum_i s_i * x_i`` in place (float32 ``h``)."""
    require_cuda(h)
    if h.dtype != torch.float32:
        raise KernelError("the residual stream is float32")
    (a, sa), (b, sb) = _terms(h, terms)
    check(fn("parallel", "sx_add_scaled")(ptr(h), ptr(a), c_int(dt_code(a.dtype) if a is not None else 0), ptr(sa), ptr(b),
                                          c_int(dt_code(b.dtype) if b is not None else 0), ptr(sb), c_int(h.shape[0]),
                                          c_int(h.shape[1]), stream()), "add_scaled")


def scale_rows(x: torch.Tensor, s: float) -> None:
    """``x *= s`` in place (float32)."""
    require_cuda(x)
    if x.dtype != torch.float32:
        raise KernelError("scale_rows takes float32")
    check(fn("parallel", "sx_scale_rows")(ptr(x), c_longlong(x.numel()), c_float(s), stream()), "scale_rows")


def side_gate(u: torch.Tensor, table: torch.Tensor, token_ids: torch.Tensor) -> torch.Tensor:
    """``gelu_tanh(u[t]) * table[id_t]`` in ``table``'s dtype: ``u`` float32 ``[T, n]``, ``table [vocab, n]``."""
    require_cuda(u, table, token_ids)
    T, n = u.shape
    if u.dtype != torch.float32 or table.shape[1] != n or token_ids.dtype != torch.int32 or token_ids.numel() != T:
        raise KernelError("side_gate: sizes or dtypes do not fit")
    g = torch.empty((T, n), dtype=table.dtype, device=u.device)
    check(fn("parallel", "sx_side_gate")(ptr(u), ptr(table), ptr(token_ids), ptr(g), c_int(T), c_int(n), c_int(table.shape[0]),
                                         c_int(dt_code(table.dtype)), stream()), "side_gate")
    return g
