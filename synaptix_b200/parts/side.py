"""A layer's own input of the token, added behind its sublayers:

    e_t = this layer's part of a row of a second token table,   y = Wp (gelu_tanh(Wg x) * e_t),   x <- x + y / rms(y) * gain

with ``x`` the residual stream after the layer's branches.  The table ``[vocab, layers * dim]`` holds the layers' parts
side by side; every layer keeps its own columns.
"""
from __future__ import annotations

from typing import Dict, List, Mapping, Optional

import torch

from .. import ops
from ..weights.loader import TensorSpec
from .base import NormedDelta, Part, Runtime, StepContext, to_device_matrix
from .linear import Linear
from .norm import RMSNorm


class TokenSide(Part):
    NAMES = {"gate": "gate", "proj": "proj", "norm": "norm"}

    def __init__(self, prefix: str, table_name: str, vocab: int, width: int, dim: int, index: int, count: int, eps: float, *,
                 names: Optional[Mapping[str, str]] = None):
        """``index`` of ``count`` parts of the table's rows belongs to this layer."""
        if not 0 <= index < count:
            raise ValueError("0 <= index < count")
        n = dict(self.NAMES, **(names or {}))
        self.table_name, self.vocab, self.width, self.dim = table_name, vocab, width, dim
        self.index, self.count = index, count
        self.gate = Linear(prefix + n["gate"], width, dim)
        self.proj = Linear(prefix + n["proj"], dim, width)
        self.norm = RMSNorm(prefix + n["norm"], width, eps)
        self.table: Optional[torch.Tensor] = None

    def children(self) -> List[Part]:
        return [self.gate, self.proj, self.norm]

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {self.table_name: TensorSpec((self.vocab, self.count * self.dim), "embedding")}

    def bind(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        self.table = to_device_matrix(tensors[self.table_name][:, self.index * self.dim:(self.index + 1) * self.dim], rt)

    def forward(self, h: torch.Tensor, terms, ctx: StepContext) -> NormedDelta:
        """Adds ``terms`` (the layer's branches, as a ``ScaledSum`` holds them) into the stream ``h`` and returns this
        input's branch, to be normed and added by whoever adds it."""
        x = ops.add_scaled_rmsnorm(h, terms, [None], 0.0, ctx.runtime.dtype)[0]
        u = self.gate.forward(x, out_dtype=torch.float32)
        g = ops.side_gate(u, self.table, ctx.token_ids)
        return NormedDelta(self.proj.forward(g), self.norm)
