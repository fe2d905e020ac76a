"""A mixer that carries a matrix per head from token to token by the gated delta rule, with a decay per key channel.

Per head ``h`` (which reads query/key head ``h // (heads / kv_heads)``), with ``q, k`` of ``dim`` and ``v`` of ``vdim``:

    q, k, v = silu(conv(Wq x)), silu(conv(Wk x)), silu(conv(Wv x)),   q, k <- u / sqrt(sum(u^2) + 1e-6),  q <- q dim^-1/2,
    b = sigmoid(Wb x),    a = exp(-exp(A_log) softplus(Wa2 (Wa1 x) + dt_bias))           (dim decays a head),
    S <- diag(a) S,   u = b (v - S^T k),   S <- S + k u^T,   o = S^T q,
    out = Wo (o / rms(o) * gain * sigmoid(Wg2 (Wg1 x)))

``conv`` is a short causal convolution over time per channel.  State of a sequence, in the cache's per-sequence storage: the
float32 matrices ``S`` (zero in a fresh slot) and a ring of the last ``taps`` projected rows for the convolutions (the row
of position ``p`` at ``p mod taps``).  Behind the projections everything on the way into ``S`` is 32-bit.
"""
from __future__ import annotations

from typing import Dict, List, Mapping, Optional

import torch

from .. import ops
from ..cache.store import BundleRequest, StateRequest
from ..weights.loader import TensorSpec
from .base import Mixer, Part, Runtime, StepContext, to_device_f32, to_device_matrix
from .linear import Linear

# single-token steps of up to this many sequences run the second halves of the low-rank projections inside the step's
# kernel (every block reads its head's rows again, from L2); larger ones as a product of their own
LOW_RANK_IN_STEP_MAX = 16


class ChannelDelta(Mixer):
    accepts_lazy_input = False
    can_defer_output = True

    NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "b": "b", "a1": "a1", "a2": "a2", "g1": "g1", "g2": "g2", "conv": ".conv",
             "a_log": "A_log", "dt_bias": "dt_bias", "norm": "norm"}
    UNIT_EPS = 1e-6                 # inside the root of q's and k's unit norms

    def __init__(self, prefix: str, width: int, heads: int, kv_heads: int, dim: int, vdim: int, *, taps: int, norm_eps: float,
                 decay_rank: Optional[int] = None, gate_rank: Optional[int] = None, q_scale: Optional[float] = None,
                 names: Optional[Mapping[str, str]] = None):
        """``decay_rank``, ``gate_rank``: sizes between the two matrices of the decays' and the output gates' projections
        (``None``: the tensors' own)."""
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if taps < 1:
            raise ValueError("a convolution has at least one tap")
        self.prefix, self.width = prefix, width
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps = heads, kv_heads, dim, vdim, taps
        self.norm_eps = float(norm_eps)
        self.decay_rank, self.gate_rank = decay_rank, gate_rank
        self.q_scale = float(q_scale) if q_scale is not None else float(dim) ** -0.5
        self.names = dict(self.NAMES, **(names or {}))
        self.channels = 2 * kv_heads * dim + heads * vdim          # convolved ones: q, k, v
        self.o = Linear(prefix + self.names["o"], heads * vdim, width)
        self.proj: Optional[torch.Tensor] = None       # [q | k | v | b | a1 | g1] stacked along the outputs
        self.low_rank: Optional[torch.Tensor] = None   # [[a2, 0], [0, g2]]
        self.consts: Optional[ops.DeltaWeights] = None
        self.ra = self.rg = 0

    def children(self) -> List[Part]:
        return [self.o]

    def _name(self, which: str) -> str:
        return self.prefix + self.names[which]

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        H, G, D, V, W = self.heads, self.kv_heads, self.dim, self.vdim, self.width
        ra = -1 if self.decay_rank is None else self.decay_rank
        rg = -1 if self.gate_rank is None else self.gate_rank
        specs = {}
        for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
            specs[self._name(n)] = TensorSpec((rows, W), "matrix")
            specs[self._name(n) + self.names["conv"]] = TensorSpec((rows, self.taps), "bias")
        specs[self._name("b")] = TensorSpec((H, W), "matrix")
        specs[self._name("a1")] = TensorSpec((ra, W), "matrix")
        specs[self._name("a2")] = TensorSpec((H * D, ra), "matrix")
        specs[self._name("g1")] = TensorSpec((rg, W), "matrix")
        specs[self._name("g2")] = TensorSpec((H * V, rg), "matrix")
        specs[self._name("a_log")] = TensorSpec((H,), "bias")
        specs[self._name("dt_bias")] = TensorSpec((H * D,), "bias")
        specs[self._name("norm")] = TensorSpec((V,), "gain")
        return specs

    def bind(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        t = {n: tensors[self._name(n)] for n in ("q", "k", "v", "b", "a1", "g1", "a2", "g2")}
        self.ra, self.rg = t["a1"].shape[0], t["g1"].shape[0]
        if t["a2"].shape[1] != self.ra or t["g2"].shape[1] != self.rg:
            raise ValueError(f"{self.prefix}: the two matrices of a low-rank projection do not share their rank")
        self.proj = to_device_matrix(torch.cat([t[n] for n in ("q", "k", "v", "b", "a1", "g1")]), rt)
        lr = torch.zeros((self.heads * (self.dim + self.vdim), self.ra + self.rg), dtype=t["a2"].dtype, device=t["a2"].device)
        lr[:self.heads * self.dim, :self.ra] = t["a2"]
        lr[self.heads * self.dim:, self.ra:] = t["g2"]
        self.low_rank = to_device_matrix(lr, rt)
        taps = torch.cat([tensors[self._name(n) + self.names["conv"]].to(torch.float32) for n in ("q", "k", "v")])
        self.consts = ops.DeltaWeights(to_device_f32(taps, rt), to_device_f32(tensors[self._name("a_log")], rt),
                                       to_device_f32(tensors[self._name("dt_bias")], rt),
                                       to_device_f32(tensors[self._name("norm")], rt))

    def cache_request(self):
        return BundleRequest((StateRequest((self.heads, self.dim, self.vdim), torch.float32),
                              StateRequest((self.taps, self.channels), torch.float32)))

    def forward(self, x: torch.Tensor, ctx: StepContext, state, write_cache: bool = True, defer_output: bool = False):
        C, H = self.channels, self.heads
        lr_col = C + H
        args = (H, self.kv_heads, self.dim, self.vdim, self.consts, self.q_scale, self.UNIT_EPS, self.norm_eps, state[0], state[1],
                ctx, x.dtype)
        if (ctx.all_single and ctx.n_seqs == x.shape[0] and x.shape[0] <= LOW_RANK_IN_STEP_MAX
                and ops.delta_step_fits(self.dim, self.vdim, self.ra, self.rg)):
            a = ops.linear(x, self.proj, out_dtype=torch.float32)
            y = ops.delta_rule(a, 0, C, *args, low_rank=self.low_rank, ra=self.ra, rg=self.rg, lr_col=lr_col)
        else:
            a = ops.linear(x, self.proj[:lr_col])                   # q, k, v and the step sizes
            z = ops.linear(ops.linear(x, self.proj[lr_col:]), self.low_rank, out_dtype=torch.float32)
            y = ops.delta_rule(a, 0, C, *args, z=z)
        if defer_output:
            return self.o.deferred(y)
        with ops.late_launch(ctx.branches):
            return self.o.forward(y)
