"""The Penopel decoder put together from parts.

A layer is a ``PreNormBlock``: ``h += mixer(norm1(h))``, then ``h += ffn(norm2(h))`` (absent where ``mlp`` is null), with norms
that compute no statistics (``DynamicTanh``), so that in bfloat16 the output product of a sublayer adds itself into the
stream and finishes the next norm on its way.  Mixers by layer type:

* ``attention``: ``Attention`` with biases on q, k and v, a rotation of the first elements of each head (``RotaryHalf``,
  optionally with frequencies scaled by bands of wavelengths, ``FrequencyBands``) and a sink of score 0 in the softmax.  A
  layer with ``kv_from`` projects queries only; its run in the schedule names the cache entry of the layer it reads;
* ``latent_attention``: ``LatentAttention`` with a query latent, neighbouring elements paired in the rotation
  (``RotaryPairs``), a window, a learned sink per head and a gate per output element.

The feed-forward is ``GeluGLU`` with biases.  The embedding's rows are multiplied by ``embedding.scale``; the logits are
capped softly in the output product.

Tensor names: ``embed``, ``head``, ``final.norm[.b|.alpha]`` and per layer ``l<i>.norm1|norm2[.b|.alpha]``, ``l<i>.mix.*``,
``l<i>.mlp.gate|up|down[.b]``.
"""
from __future__ import annotations

from ..config.penopel import PenopelConfig
from ..config.registry import register_architecture
from ..parts import (Attention, DynamicTanh, Embedding, FrequencyBands, GeluGLU, LatentAttention, NoPosition, OutputHead,
                     PreNormBlock, RotaryHalf, RotaryPairs)
from .decoder import DecoderModel, LayerRun

ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o"}
FF_NAMES = {"gate": "gate", "up": "up", "down": "down"}
BIAS_SUFFIX = ".b"
SINK_SCORE = 0.0            # an attention layer's softmax has one more term, exp(0), in its denominator


def _position(cls, head_dim: int, rot):
    if rot is None:
        return NoPosition()
    bands = None if rot.factor is None else FrequencyBands(rot.factor, rot.low, rot.high, rot.original)
    return cls(head_dim, rot.base, rotary_dim=rot.dims, scaling=bands)


def build_penopel(cfg: PenopelConfig) -> DecoderModel:
    W = cfg.width
    embedding = Embedding("embed", cfg.vocab, W, scale=cfg.embedding_scale)
    layers, schedule, entry_of = [], [], {}
    for i, spec in enumerate(cfg.layers):
        p = f"l{i}."
        source = None
        if spec.type == "attention":
            a = spec.attention
            source = a.kv_from
            mixer = Attention(p + "mix.", W, a.heads, a.kv_heads, a.dim, position=_position(RotaryHalf, a.dim, a.rot), scale=a.scale,
                              v_head_dim=a.vdim, sink_score=SINK_SCORE, bias_suffix=BIAS_SUFFIX, own_kv=source is None,
                              names=ATTENTION_NAMES)
        else:
            a = spec.latent
            mixer = LatentAttention(p + "mix.", W, a.heads, a.dim, a.rot_dim, a.vdim, a.q_rank, a.kv_rank, scale=a.scale,
                                    position=_position(RotaryPairs, a.rot_dim, a.rot), norm_eps=cfg.norm_eps, window=a.window,
                                    gated="elements", sinks=True)
        norm2 = ffn = None
        if spec.ff is not None:
            norm2, ffn = DynamicTanh(p + "norm2", W), GeluGLU(p + "mlp.", W, spec.ff, names=FF_NAMES, bias_suffix=BIAS_SUFFIX)
        layers.append(PreNormBlock(DynamicTanh(p + "norm1", W), mixer, norm2, ffn))
        if source is not None:
            schedule.append(LayerRun(i, entry_of[source], write_cache=False))
        else:
            entry_of[i] = len(entry_of)
            schedule.append(LayerRun(i, entry_of[i]))
    return DecoderModel(cfg, embedding, layers, DynamicTanh("final.norm", W),
                        OutputHead("head", cfg.vocab, W, False, embedding, softcap=cfg.logit_softcap), schedule=schedule)


register_architecture(PenopelConfig, build_penopel)
