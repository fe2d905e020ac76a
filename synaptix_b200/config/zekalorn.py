"""Typed configuration of the Zekalorn decoder, read from its config.json.

Keys: ``architecture`` ("Zekalorn"), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (the embedding's rows are
multiplied by it), ``max_positions`` (rows of the learned position table; a sequence can be no longer), ``token_side.dim``
(elements a layer takes of the second token table; absent: no layer has a token input of its own), ``loop`` (``start``,
``stop``, ``times``: layers ``start .. stop-1`` run ``times`` times in a row with the same weights; absent: every layer
runs once) and ``layers`` (a list; each entry has ``type``, the sizes of its mixer under ``mixer`` and its feed-forward
under ``mlp`` or ``null``).  Layer types:

* ``channel_delta``: a gated delta rule with a decay per key channel: ``heads`` (values, decays), ``kv_heads`` (queries and
  keys), ``dim``, ``vdim``, ``conv`` (taps of the short convolutions).  The ranks of the two low-rank projections are the
  tensors' own sizes, which ``decay_rank`` and ``gate_rank`` may state for a model whose weights are yet to be made;
* ``attention``: grouped-query softmax attention without rotation: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``,
  ``bias_max`` (the distance at which the logarithmic buckets of the learned distance bias end; the number of buckets is
  the table's own first size, which ``bias_rows`` may state) and ``q_temp`` (``coef``, ``every``: queries are multiplied
  by ``1 + coef ln(floor((p + 1) / every) + 1)`` at position ``p``; absent: not at all).

Feed-forward: ``mlp.kind`` = ``dense`` with ``ff``, or ``moe`` with ``expert.ff``, ``router.experts``, ``router.top``.
Every size and constant is taken from here; a key that is required and missing, or a type or kind that is not known, is
an error.
"""
from __future__ import annotations

import dataclasses
from typing import Any, ClassVar, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, take


@dataclasses.dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: Optional[int] = None         # None: the tensor's own size
    gate_rank: Optional[int] = None

    @classmethod
    def from_dict(cls, d, where):
        return cls(heads=take(d, "heads", int, where=where), kv_heads=take(d, "kv_heads", int, where=where),
                   dim=take(d, "dim", int, where=where), vdim=take(d, "vdim", int, where=where),
                   conv=take(d, "conv", int, where=where), decay_rank=take(d, "decay_rank", int, None, where=where),
                   gate_rank=take(d, "gate_rank", int, None, where=where))

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}
        if self.decay_rank is not None:
            d["decay_rank"] = self.decay_rank
        if self.gate_rank is not None:
            d["gate_rank"] = self.gate_rank
        return d

    def validate(self, where):
        if min(self.heads, self.kv_heads, self.dim, self.vdim, self.conv) <= 0 or self.heads % self.kv_heads:
            raise ConfigError(f"{where}: heads must be a positive multiple of kv_heads, dim, vdim and conv positive")
        for r in (self.decay_rank, self.gate_rank):
            if r is not None and r <= 0:
                raise ConfigError(f"{where}: decay_rank and gate_rank must be > 0")


@dataclasses.dataclass(frozen=True)
class BiasedAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    bias_rows: Optional[int] = None          # rows of the distance table; None: the tensor's own size
    temp_coef: Optional[float] = None        # both constants of the temperature, or both None
    temp_every: Optional[int] = None

    @classmethod
    def from_dict(cls, d, where):
        temp = d.get("q_temp")
        kw = {}
        if temp is not None:
            if not isinstance(temp, dict):
                raise ConfigError(f"{where}: 'q_temp' must be an object or null")
            kw = dict(temp_coef=take(temp, "coef", float, where=where + ".q_temp"),
                      temp_every=take(temp, "every", int, where=where + ".q_temp"))
        return cls(heads=take(d, "heads", int, where=where), kv_heads=take(d, "kv_heads", int, where=where),
                   dim=take(d, "dim", int, where=where), vdim=take(d, "vdim", int, where=where),
                   scale=take(d, "scale", float, where=where), bias_max=take(d, "bias_max", float, where=where),
                   bias_rows=take(d, "bias_rows", int, None, where=where), **kw)

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "bias_max": self.bias_max}
        if self.bias_rows is not None:
            d["bias_rows"] = self.bias_rows
        if self.temp_coef is not None:
            d["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return d

    def validate(self, where):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) <= 0 or self.heads % self.kv_heads:
            raise ConfigError(f"{where}: heads must be a positive multiple of kv_heads, dim and vdim positive")
        if self.bias_max <= 0:
            raise ConfigError(f"{where}: bias_max must be > 0")
        if self.bias_rows is not None and self.bias_rows < 2:
            raise ConfigError(f"{where}: bias_rows must be at least 2")
        if self.temp_every is not None and self.temp_every <= 0:
            raise ConfigError(f"{where}: q_temp.every must be > 0")


@dataclasses.dataclass(frozen=True)
class FeedForwardSpec:
    kind: str                                # "dense" or "moe"
    ff: int
    experts: int = 0
    top: int = 0

    @classmethod
    def from_dict(cls, d, where):
        kind = take(d, "kind", str, where=where)
        if kind == "dense":
            return cls(kind=kind, ff=take(d, "ff", int, where=where))
        if kind != "moe":
            raise ConfigError(f"{where}: unknown kind {kind!r} (known: dense, moe)")
        expert, router = d.get("expert"), d.get("router")
        if not isinstance(expert, dict) or not isinstance(router, dict):
            raise ConfigError(f"{where}: 'expert' and 'router' must be objects")
        return cls(kind=kind, ff=take(expert, "ff", int, where=where + ".expert"),
                   experts=take(router, "experts", int, where=where + ".router"),
                   top=take(router, "top", int, where=where + ".router"))

    def to_dict(self):
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}

    def validate(self, where):
        if self.ff <= 0:
            raise ConfigError(f"{where}: ff must be > 0")
        if self.kind == "moe" and not (0 < self.top <= self.experts):
            raise ConfigError(f"{where}: 0 < router.top <= router.experts")


@dataclasses.dataclass(frozen=True)
class ZekalornLayer:
    type: str
    delta: Optional[DeltaSpec] = None
    attention: Optional[BiasedAttentionSpec] = None
    mlp: Optional[FeedForwardSpec] = None    # None: the layer has no feed-forward

    @classmethod
    def from_dict(cls, d, i):
        where = f"config.json: layers[{i}]"
        if not isinstance(d, dict):
            raise ConfigError(f"{where} must be an object")
        typ = take(d, "type", str, where=where)
        mixer = d.get("mixer")
        if not isinstance(mixer, dict):
            raise ConfigError(f"{where}: 'mixer' must be an object")
        kw: Dict[str, Any] = {}
        if typ == "channel_delta":
            kw["delta"] = DeltaSpec.from_dict(mixer, where + ".mixer")
        elif typ == "attention":
            kw["attention"] = BiasedAttentionSpec.from_dict(mixer, where + ".mixer")
        else:
            raise ConfigError(f"{where}: unknown layer type {typ!r} (known: channel_delta, attention)")
        mlp = d.get("mlp")
        if mlp is not None:
            if not isinstance(mlp, dict):
                raise ConfigError(f"{where}: 'mlp' must be an object or null")
            kw["mlp"] = FeedForwardSpec.from_dict(mlp, where + ".mlp")
        return cls(type=typ, **kw)

    def to_dict(self):
        mixer = self.delta.to_dict() if self.type == "channel_delta" else self.attention.to_dict()
        return {"type": self.type, "mixer": mixer, "mlp": None if self.mlp is None else self.mlp.to_dict()}

    def validate(self, i):
        where = f"config.json: layers[{i}]"
        (self.delta or self.attention).validate(where + ".mixer")
        if self.mlp is not None:
            self.mlp.validate(where + ".mlp")


@dataclasses.dataclass(frozen=True)
class ZekalornConfig(ModelConfig):
    architectures: ClassVar[Tuple[str, ...]] = ("Zekalorn",)
    model_types: ClassVar[Tuple[str, ...]] = ("zekalorn",)

    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    max_positions: int = 0
    side_dim: Optional[int] = None           # None: no token input per layer
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    has_loop: bool = False
    layers: Tuple[ZekalornLayer, ...] = ()

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ZekalornConfig":
        norm, emb = d.get("norm"), d.get("embedding")
        if not isinstance(norm, dict) or not isinstance(emb, dict):
            raise ConfigError("config.json: 'norm' and 'embedding' must be objects")
        layers, loop, side = d.get("layers"), d.get("loop"), d.get("token_side")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        kw: Dict[str, Any] = {}
        if loop is not None:
            if not isinstance(loop, dict):
                raise ConfigError("config.json: 'loop' must be an object or null")
            kw.update(loop_start=take(loop, "start", int, where="config.json: loop"),
                      loop_stop=take(loop, "stop", int, where="config.json: loop"),
                      loop_times=take(loop, "times", int, where="config.json: loop"), has_loop=True)
        if side is not None:
            if not isinstance(side, dict):
                raise ConfigError("config.json: 'token_side' must be an object or null")
            kw["side_dim"] = take(side, "dim", int, where="config.json: token_side")
        cfg = cls(vocab=take(d, "vocab", int), width=take(d, "width", int),
                  norm_eps=take(norm, "eps", float, where="config.json: norm"),
                  embedding_scale=take(emb, "scale", float, where="config.json: embedding"),
                  max_positions=take(d, "max_positions", int),
                  layers=tuple(ZekalornLayer.from_dict(x, i) for i, x in enumerate(layers)), **kw)
        cfg.validate()
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architectures[0], "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
             "max_positions": self.max_positions, "layers": [x.to_dict() for x in self.layers]}
        if self.side_dim is not None:
            d["token_side"] = {"dim": self.side_dim}
        if self.has_loop:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return d

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.max_positions <= 0:
            raise ConfigError("config.json: vocab, width and max_positions must be > 0")
        if self.norm_eps < 0:
            raise ConfigError("config.json: norm.eps must be >= 0")
        if self.side_dim is not None and self.side_dim <= 0:
            raise ConfigError("config.json: token_side.dim must be > 0")
        for i, layer in enumerate(self.layers):
            layer.validate(i)
        if self.has_loop:
            if not (0 <= self.loop_start <= self.loop_stop <= len(self.layers)) or self.loop_times < 1:
                raise ConfigError("config.json: loop needs 0 <= start <= stop <= number of layers and times >= 1")

    def runs(self):
        """The order in which layers run: ``(layer, pass)`` with ``pass`` the number of the loop's pass that the run
        opens, else ``None``."""
        if not self.has_loop or self.loop_start == self.loop_stop:
            return [(i, None) for i in range(len(self.layers))]
        out = [(i, None) for i in range(self.loop_start)]
        for t in range(self.loop_times):
            out += [(i, t if i == self.loop_start else None) for i in range(self.loop_start, self.loop_stop)]
        return out + [(i, None) for i in range(self.loop_stop, len(self.layers))]
