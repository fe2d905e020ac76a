"""Typed configuration of the Penopel decoder, read from its config.json.

Keys: ``architecture`` ("Penopel"), ``vocab``, ``width``, ``norm.eps`` (of the norms inside latent attention),
``embedding.scale``, ``logit_softcap`` (absent or 0: the logits are not capped) and ``layers`` (a list; each entry has
``type``, the sizes of its mixer under ``mixer`` and its feed-forward under ``mlp`` or ``null``).  Layer types:

* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot`` (``dims``, ``base`` and optionally ``scaling``
  with ``factor``, ``low``, ``high``, ``original``; absent: no rotation) and optionally ``kv_from``, the earlier layer whose
  keys and values it reads;
* ``latent_attention``: ``heads``, ``dim`` (unrotated query/key elements a head), ``rot_dim`` (rotated ones, the key's shared
  by all heads), ``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot`` (as above) and ``mask.size`` (the window; absent: every
  earlier key is seen).

Feed-forward: ``mlp.kind`` = ``dense`` with ``ff``.  Every size and constant is taken from here; a key that is required and
missing, or a type or kind that is not known, is an error.
"""
from __future__ import annotations

import dataclasses
from typing import Any, ClassVar, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, take


def _obj(d, key, where, required=True):
    v = d.get(key)
    if v is None and not required:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: '{key}' must be an object")
    return v


@dataclasses.dataclass(frozen=True)
class RotationSpec:
    dims: int
    base: float
    factor: Optional[float] = None      # the four numbers of the frequency bands come together or not at all
    low: Optional[float] = None
    high: Optional[float] = None
    original: Optional[float] = None

    @classmethod
    def from_dict(cls, d, where):
        sc = _obj(d, "scaling", where, required=False)
        kw = {}
        if sc is not None:
            kw = {k: take(sc, k, float, where=where + ".scaling") for k in ("factor", "low", "high", "original")}
        return cls(dims=take(d, "dims", int, where=where), base=take(d, "base", float, where=where), **kw)

    def to_dict(self):
        d = {"dims": self.dims, "base": self.base}
        if self.factor is not None:
            d["scaling"] = {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}
        return d

    def validate(self, limit, where):
        if self.dims % 2 or not (0 < self.dims <= limit) or self.base <= 0:
            raise ConfigError(f"{where}: rot.dims must be even and at most {limit}, rot.base positive")
        if self.factor is not None and (min(self.factor, self.low, self.original) <= 0 or self.high < self.low):
            raise ConfigError(f"{where}: rot.scaling needs positive numbers and high >= low")


@dataclasses.dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationSpec] = None
    kv_from: Optional[int] = None

    @classmethod
    def from_dict(cls, d, where):
        rot = _obj(d, "rot", where, required=False)
        return cls(heads=take(d, "heads", int, where=where), kv_heads=take(d, "kv_heads", int, where=where),
                   dim=take(d, "dim", int, where=where), vdim=take(d, "vdim", int, where=where),
                   scale=take(d, "scale", float, where=where),
                   rot=None if rot is None else RotationSpec.from_dict(rot, where + ".rot"),
                   kv_from=take(d, "kv_from", int, None, where=where))

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d

    def validate(self, where):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) <= 0 or self.heads % self.kv_heads or self.scale <= 0:
            raise ConfigError(f"{where}: heads, kv_heads, dim, vdim and scale must be > 0, heads a multiple of kv_heads")
        if self.rot is not None:
            self.rot.validate(self.dim, where)


@dataclasses.dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Optional[RotationSpec] = None
    window: Optional[int] = None

    @classmethod
    def from_dict(cls, d, where):
        rot = _obj(d, "rot", where, required=False)
        mask = d.get("mask") or {}
        return cls(heads=take(d, "heads", int, where=where), dim=take(d, "dim", int, where=where),
                   rot_dim=take(d, "rot_dim", int, where=where), vdim=take(d, "vdim", int, where=where),
                   q_rank=take(d, "q_rank", int, where=where), kv_rank=take(d, "kv_rank", int, where=where),
                   scale=take(d, "scale", float, where=where),
                   rot=None if rot is None else RotationSpec.from_dict(rot, where + ".rot"),
                   window=take(mask, "size", int, None, where=where + ".mask"))

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
             "kv_rank": self.kv_rank, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d

    def validate(self, where):
        if min(self.heads, self.vdim, self.q_rank, self.kv_rank, self.rot_dim) <= 0 or self.dim < 0 or self.scale <= 0:
            raise ConfigError(f"{where}: heads, rot_dim, vdim, q_rank, kv_rank and scale must be > 0")
        if self.window is not None and self.window <= 0:
            raise ConfigError(f"{where}: mask.size must be > 0")
        if self.rot is not None:
            self.rot.validate(self.rot_dim, where)


@dataclasses.dataclass(frozen=True)
class PenopelLayer:
    type: str
    attention: Optional[AttentionSpec] = None
    latent: Optional[LatentSpec] = None
    ff: Optional[int] = None                    # None: the layer has no feed-forward

    @classmethod
    def from_dict(cls, d, i):
        where = f"config.json: layers[{i}]"
        if not isinstance(d, dict):
            raise ConfigError(f"{where} must be an object")
        typ = take(d, "type", str, where=where)
        mixer = _obj(d, "mixer", where)
        kw: Dict[str, Any] = {}
        if typ == "attention":
            kw["attention"] = AttentionSpec.from_dict(mixer, where + ".mixer")
        elif typ == "latent_attention":
            kw["latent"] = LatentSpec.from_dict(mixer, where + ".mixer")
        else:
            raise ConfigError(f"{where}: unknown layer type {typ!r} (known: attention, latent_attention)")
        mlp = _obj(d, "mlp", where, required=False)
        if mlp is not None:
            kind = take(mlp, "kind", str, where=where + ".mlp")
            if kind != "dense":
                raise ConfigError(f"{where}.mlp: unknown kind {kind!r} (known: dense)")
            kw["ff"] = take(mlp, "ff", int, where=where + ".mlp")
        return cls(type=typ, **kw)

    def to_dict(self):
        mixer = self.attention.to_dict() if self.type == "attention" else self.latent.to_dict()
        return {"type": self.type, "mixer": mixer, "mlp": None if self.ff is None else {"kind": "dense", "ff": self.ff}}


@dataclasses.dataclass(frozen=True)
class PenopelConfig(ModelConfig):
    architectures: ClassVar[Tuple[str, ...]] = ("Penopel",)
    model_types: ClassVar[Tuple[str, ...]] = ("penopel",)

    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    logit_softcap: Optional[float] = None
    layers: Tuple[PenopelLayer, ...] = ()

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PenopelConfig":
        norm, emb = _obj(d, "norm", "config.json"), _obj(d, "embedding", "config.json")
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        cfg = cls(vocab=take(d, "vocab", int), width=take(d, "width", int),
                  norm_eps=take(norm, "eps", float, where="config.json: norm"),
                  embedding_scale=take(emb, "scale", float, where="config.json: embedding"),
                  logit_softcap=take(d, "logit_softcap", float, None) or None,
                  layers=tuple(PenopelLayer.from_dict(x, i) for i, x in enumerate(layers)))
        cfg.validate()
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architectures[0], "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale}, "layers": [x.to_dict() for x in self.layers]}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("config.json: vocab and width must be > 0")
        if self.norm_eps < 0:
            raise ConfigError("config.json: norm.eps must be >= 0")
        if self.logit_softcap is not None and self.logit_softcap <= 0:
            raise ConfigError("config.json: logit_softcap must be > 0")
        for i, layer in enumerate(self.layers):
            where = f"config.json: layers[{i}]"
            (layer.attention or layer.latent).validate(where + ".mixer")
            if layer.ff is not None and layer.ff <= 0:
                raise ConfigError(f"{where}.mlp: ff must be > 0")
            if layer.type == "attention" and layer.attention.kv_from is not None:
                j = layer.attention.kv_from
                src = self.layers[j].attention if 0 <= j < i else None
                if src is None or src.kv_from is not None:
                    raise ConfigError(f"{where}: kv_from must name an earlier attention layer with keys and values of its own")
                a = layer.attention
                if (a.heads, a.kv_heads, a.dim, a.vdim, a.rot) != (src.heads, src.kv_heads, src.dim, src.vdim, src.rot):
                    raise ConfigError(f"{where}: the layer it reads keys and values from has other head counts, sizes or rotation")
