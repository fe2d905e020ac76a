"""Matrix products ``y = x W^T`` with weight ``[out, in]``, by default without bias
(crates/synaptix-nn/src/linear.rs:10-35; the Qwen3 decoder binds every projection
without bias, crates/synaptix-models/llm/common/src/weights.rs:49-51).  With
``bias_suffix`` every named matrix has a vector of that name with the suffix added,
which joins the product (32-bit) ahead of its epilogue.  ``row_order`` gives named
matrices (and their biases) another order of rows when they are bound.

``Linear`` may bind several named matrices and stack them along the output
dimension, so that q/k/v (or gate/up) become one product; the checkpoint keeps
its separate tensors and names.  ``JoinedLinear`` stacks along the INPUT
dimension instead: the sum of several products ``sum_i x_i W_i^T`` as one
product over the concatenated inputs.
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional, Sequence

import torch

from .. import ops
from ..weights.loader import TensorSpec
from .base import Part, PendingLinear, PendingNorm, Runtime, ScaledRows, to_device_f32, to_device_matrix


class Linear(Part):
    def __init__(self, weight_names: Sequence[str], in_features: int, out_features: Sequence[int],
                 kind: str = "matrix", bias_suffix: Optional[str] = None,
                 row_order: Optional[Mapping[str, torch.Tensor]] = None):
        if isinstance(weight_names, str):
            weight_names = [weight_names]
            out_features = [out_features]
        self.weight_names = list(weight_names)
        self.in_features = in_features
        self.out_features = list(out_features)
        self.kind = kind
        self.bias_suffix = bias_suffix
        self.row_order = dict(row_order or {})
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None        # float32 [total_out]

    @property
    def total_out(self) -> int:
        return sum(self.out_features)

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        specs = {n: TensorSpec((o, self.in_features), self.kind)
                 for n, o in zip(self.weight_names, self.out_features)}
        if self.bias_suffix is not None:
            specs.update({n + self.bias_suffix: TensorSpec((o,), "bias") for n, o in zip(self.weight_names, self.out_features)})
        return specs

    def _ordered(self, tensors: Mapping[str, torch.Tensor], n: str, suffix: str = "") -> torch.Tensor:
        t, order = tensors[n + suffix], self.row_order.get(n)
        return t if order is None else t[order.to(t.device)]

    def bind(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        ws = [to_device_matrix(self._ordered(tensors, n), rt) for n in self.weight_names]
        self.weight = ws[0] if len(ws) == 1 else torch.cat(ws, dim=0).contiguous()
        if self.bias_suffix is not None:
            self.bias = to_device_f32(torch.cat([self._ordered(tensors, n, self.bias_suffix).to(torch.float32)
                                                 for n in self.weight_names]), rt)

    def share(self, weight: torch.Tensor) -> None:
        """Use an already bound matrix (a tied output head uses the embedding table)."""
        self.weight = weight

    def deferred(self, x: torch.Tensor) -> PendingLinear:
        """This product, not run yet (see ``PendingLinear``)."""
        return PendingLinear(x, self.weight, self.bias)

    def forward(self, x: torch.Tensor, out_dtype: Optional[torch.dtype] = None,
                epilogue: Optional[str] = None, cap: float = 0.0) -> torch.Tensor:
        """``cap > 0`` (float32 results): ``cap * tanh(. / cap)`` of them, in the product's epilogue."""
        if (self.bias is not None or cap) and not isinstance(x, torch.Tensor):
            x = x.materialize()            # the forms that norm on the way take neither
        if isinstance(x, ScaledRows):
            y = ops.linear_scaled(x.x, x.ssq, x.eps, self.weight, out_dtype=out_dtype, epilogue=epilogue)
            if y is not None:
                return y
            x = x.materialize()
        if isinstance(x, PendingNorm):
            y = ops.linear_normed(x, self.weight, out_dtype=out_dtype, epilogue=epilogue)
            if y is not None:
                return y
            x = x.materialize()
        return ops.linear(x, self.weight, out_dtype=out_dtype, epilogue=epilogue, bias=self.bias, cap=cap)


class JoinedLinear(Linear):
    """``[x_1 | x_2 | ...] @ [W_1 | W_2 | ...].T = sum_i x_i W_i^T``: named matrices ``[out, in_i]`` stacked along their
    inputs, so that branches that are added after their output projections share one product."""

    def __init__(self, weight_names: Sequence[str], in_features: Sequence[int], out_features: int):
        self.weight_names = list(weight_names)
        self.in_parts = list(in_features)
        self.in_features = sum(self.in_parts)
        self.out_features = [out_features]
        self.kind = "matrix"
        self.bias_suffix, self.row_order = None, {}
        self.weight = self.bias = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {n: TensorSpec((self.out_features[0], i), self.kind) for n, i in zip(self.weight_names, self.in_parts)}

    def bind(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        ws = [to_device_matrix(tensors[n], rt) for n in self.weight_names]
        self.weight = ws[0] if len(ws) == 1 else torch.cat(ws, dim=1).contiguous()
