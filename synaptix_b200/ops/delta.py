"""Python face of the kernels in ``csrc/delta.cu``: the gated delta rule with a decay per key channel, its short
convolutions, unit norms, step sizes, decays and output gate."""
from __future__ import annotations

from typing import NamedTuple, Optional

import torch

from ._lib import KernelError, c_float, c_int, check, dt_code, fn, late_launch, ptr, require_cuda, stream

# portions of at least this many tokens (the longest of a step) run in chunks; shorter ones walk the tokens
CHUNKS_MIN_TOKENS = 16

_CHUNK = [0]


class DeltaWeights(NamedTuple):
    """What the recurrence needs beside the projections: ``taps`` float32 ``[2 kv_heads dim + heads vdim, n]`` (q, k, v
    channels), ``a_log`` float32 ``[heads]``, ``dt_bias`` float32 ``[heads dim]``, ``gain`` float32 ``[vdim]``."""
    taps: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    gain: torch.Tensor


def delta_step_fits(dim: int, vdim: int, ra: int, rg: int) -> bool:
    """Whether single-token steps of these head sizes run as one kernel (``ra``, ``rg``: ranks of the two low-rank
    projections, 0 where their results are handed over formed)."""
    return bool(fn("delta", "sx_delta_step_fits")(c_int(dim), c_int(vdim), c_int(ra), c_int(rg)))


def delta_rule(proj: torch.Tensor, col: int, b_col: int, heads: int, kv_heads: int, dim: int, vdim: int, w: DeltaWeights,
               q_scale: float, unit_eps: float, eps: float, S: torch.Tensor, hist: torch.Tensor, ctx, out_dtype: torch.dtype,
               *, z: Optional[torch.Tensor] = None, low_rank: Optional[torch.Tensor] = None, ra: int = 0, rg: int = 0,
               lr_col: int = 0) -> torch.Tensor:
    """The recurrence over the step's tokens (see ``csrc/delta.cu``): ``[T, heads * vdim]`` in ``out_dtype``.

    ``proj [T, row]`` holds q, k (``kv_heads * dim`` columns each), v (``heads * vdim``) from ``col`` on and the step sizes'
    pre-activations (``heads``) from ``b_col`` on.  ``z`` float32 ``[T, heads * dim + heads * vdim]``: the decays' and the
    output gates' pre-activations; or, in single-token steps, ``low_rank`` (compute dtype
    ``[heads * dim + heads * vdim, ra + rg]``, block-diagonal) and the columns ``lr_col ..`` of ``proj`` it is applied to.
    ``S`` float32 ``[slots, heads, dim, vdim]`` and ``hist`` float32 ``[slots, taps, channels]`` are moved on."""
    require_cuda(proj, w.taps, w.a_log, w.dt_bias, w.gain, S, hist, z, low_rank)
    T, row = proj.shape
    C = 2 * kv_heads * dim + heads * vdim
    taps = w.taps.shape[1]
    for t in (w.taps, w.a_log, w.dt_bias, w.gain, S, hist, z):
        if t is not None and t.dtype != torch.float32:
            raise KernelError("delta_rule: taps, decays' constants, gains, pre-activations and states are float32")
    if (heads % kv_heads or w.taps.shape[0] != C or w.a_log.numel() != heads or w.dt_bias.numel() != heads * dim
            or w.gain.numel() != vdim or tuple(S.shape[1:]) != (heads, dim, vdim) or tuple(hist.shape[1:]) != (taps, C)
            or col + C > row or b_col + heads > row):
        raise KernelError("delta_rule: the constants, states or columns do not fit the heads")
    nz = heads * (dim + vdim)
    if (z is None) == (low_rank is None):
        raise KernelError("delta_rule: pre-activations, or the low-rank matrices that give them")
    if z is not None and tuple(z.shape) != (T, nz):
        raise KernelError("delta_rule: the pre-activations do not fit the heads")
    if low_rank is not None and (tuple(low_rank.shape) != (nz, ra + rg) or lr_col + ra + rg > row or low_rank.dtype != out_dtype):
        raise KernelError("delta_rule: the low-rank matrices do not fit")
    out = torch.empty((T, heads * vdim), dtype=out_dtype, device=proj.device)

    def common():
        return (ptr(proj), c_int(row), c_int(col), c_int(b_col), ptr(w.taps), c_int(taps), ptr(hist), ptr(z), c_int(nz), ptr(w.a_log),
                ptr(w.dt_bias), ptr(w.gain), c_float(q_scale), c_float(unit_eps), c_float(eps), ptr(S), ptr(out), ptr(ctx.positions),
                ptr(ctx.seq_of_token), ptr(ctx.cu_seqlens), ptr(ctx.seq_past), ptr(ctx.seq_lens), ptr(ctx.seq_slots), c_int(T),
                c_int(ctx.n_seqs), c_int(heads), c_int(kv_heads), c_int(dim), c_int(vdim), c_int(dt_code(proj.dtype)),
                c_int(dt_code(out_dtype)))

    single = ctx.all_single and ctx.n_seqs == T
    if single and delta_step_fits(dim, vdim, ra if low_rank is not None else 0, rg if low_rank is not None else 0):
        check(fn("delta", "sx_delta_step")(*common(), ptr(low_rank), c_int(ra), c_int(rg), c_int(lr_col), stream()), "delta_step")
        return out
    if low_rank is not None:
        raise KernelError("delta_rule: the low-rank matrices are applied by the single-token kernel only (ask delta_step_fits)")
    f32 = dict(dtype=torch.float32, device=proj.device)
    q = torch.empty((T, kv_heads * dim), **f32)
    k = torch.empty_like(q)
    v = torch.empty((T, heads * vdim), **f32)
    check(fn("delta", "sx_delta_prepare")(*common(), ptr(q), ptr(k), ptr(v), stream()), "delta_prepare", launches=2)
    if ctx.max_new >= CHUNKS_MIN_TOKENS and fn("delta", "sx_delta_chunks_fit")(c_int(dim), c_int(vdim)):
        if _CHUNK[0] == 0:
            _CHUNK[0] = int(fn("delta", "sx_delta_chunk_tokens")())
        C_ = _CHUNK[0]
        chunks = (ctx.max_new + C_ - 1) // C_
        n = (T // C_ + ctx.n_seqs) * heads
        x, qg, kd = (torch.empty((n, C_, dim), **f32) for _ in range(3))
        y, p, ge = torch.empty((n, C_, vdim), **f32), torch.empty((n, C_, C_), **f32), torch.empty((n, dim), **f32)
        sb = torch.empty((n, dim, vdim), **f32)
        # columns of the state a block of the scan owns: narrow slices where wide ones would leave SMs idle (every slice
        # reads the chunks' keys again)
        sms = torch.cuda.get_device_properties(proj.device).multi_processor_count
        blocks = ctx.n_seqs * heads
        slice_ = next((v for v in (32, 16) if blocks * ((vdim + v - 1) // v) >= 0.8 * sms), 8)
        # each of the three fills the SMs' shared memory: waiting blocks of the next would only take the running one's room
        # (16 heads of 128 x 128, 2,048 tokens: 447 us scheduled early, 365 late)
        with late_launch():
            check(fn("delta", "sx_delta_chunks")(*common(), ptr(q), ptr(k), ptr(v), ptr(x), ptr(qg), ptr(kd), ptr(y), ptr(p), ptr(ge),
                                                 ptr(sb), c_int(chunks), c_int(slice_), stream()), "delta_chunks", launches=3)
    else:
        check(fn("delta", "sx_delta_walk")(*common(), ptr(q), ptr(k), ptr(v), stream()), "delta_walk")
    return out
