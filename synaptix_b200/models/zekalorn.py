"""The Zekalorn decoder put together from parts.

The embedding's rows are multiplied by ``embedding.scale`` and a learned vector of the position is added.  A layer is a
``ParallelBlock`` with ONE norm that both sublayers read, ``h += mixer(norm1(h)) + ff(norm1(h))``, and an input of the token
of its own behind the sum (``TokenSide``).  Mixers by layer type:

* ``channel_delta``: ``ChannelDelta``, a gated delta rule with a decay per key channel behind short convolutions;
* ``attention``: ``ScoredAttention`` with softmax weights, a learned bias per head and distance bucket, and queries that are
  multiplied by a temperature of their position.

Feed-forwards: ``SwiGLU`` (dense) or ``MixtureOfExperts`` whose weights are the softmax over the chosen logits (the softmax
over all of them, divided by the sum of the chosen) and whose experts have no gate (``relu(.)^2``).

A stretch of layers may run several times with the same weights (``loop``): every pass has cache entries of its own, and
before every pass a learned vector of that pass (``loop.step[t]``) is added to the stream.

Tensor names: ``embed``, ``pos``, ``side.embed``, ``loop.step``, ``head``, ``final.norm``, and per layer ``l<i>.norm1``,
``l<i>.mix.*``, ``l<i>.mlp.gate|up|down`` or ``l<i>.mlp.router|e<j>.up|e<j>.down``, ``l<i>.side.gate|proj|norm``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zekalorn import ZekalornConfig
from ..parts import (ChannelDelta, Embedding, MixtureOfExperts, OutputHead, ParallelBlock, RMSNorm, ScoredAttention, SwiGLU,
                     TokenSide)
from .decoder import DecoderModel, Inject, LayerRun, StreamVectors


def build_zekalorn(cfg: ZekalornConfig) -> DecoderModel:
    W, eps, n = cfg.width, cfg.norm_eps, len(cfg.layers)
    embedding = Embedding("embed", cfg.vocab, W, scale=cfg.embedding_scale, positions=("pos", cfg.max_positions))
    layers = []
    for i, spec in enumerate(cfg.layers):
        p = f"l{i}."
        if spec.type == "channel_delta":
            m = spec.delta
            mixer = ChannelDelta(p + "mix.", W, m.heads, m.kv_heads, m.dim, m.vdim, taps=m.conv, norm_eps=eps,
                                 decay_rank=m.decay_rank, gate_rank=m.gate_rank)
        else:
            m = spec.attention
            mixer = ScoredAttention(p + "mix.", W, m.heads, m.kv_heads, m.dim, m.vdim, scale=m.scale, weights="softmax",
                                    distance_bias=(m.bias_rows, m.bias_max),
                                    q_temp=None if m.temp_coef is None else (m.temp_coef, m.temp_every))
        ffn = None
        if spec.mlp is not None:
            f = spec.mlp
            if f.kind == "dense":
                ffn = SwiGLU(p + "mlp.", W, f.ff, names={"gate": "gate", "up": "up", "down": "down"})
            else:
                ffn = MixtureOfExperts(p + "mlp.", W, f.ff, f.experts, f.top, gated=False)
        side = None
        if cfg.side_dim is not None:
            side = TokenSide(p + "side.", "side.embed", cfg.vocab, W, cfg.side_dim, i, n, eps)
        layers.append(ParallelBlock(RMSNorm(p + "norm1", W, eps), mixer, None, ffn, side=side))
    schedule = []
    for entry, (layer, opens_pass) in enumerate(cfg.runs()):
        if opens_pass is not None:
            schedule.append(Inject(row=opens_pass))
        schedule.append(LayerRun(layer, entry))
    vectors = StreamVectors("loop.step", cfg.loop_times, W) if cfg.has_loop else None
    return DecoderModel(cfg, embedding, layers, RMSNorm("final.norm", W, eps),
                        OutputHead("head", cfg.vocab, W, False, embedding), schedule=schedule, stream_vectors=vectors)


register_architecture(ZekalornConfig, build_zekalorn)
