"""Ranilix's configuration, read from the keys of its config.json.

Top level: ``architecture`` ("Ranilix"), ``vocab``, ``width``, ``embedding.scale`` (absent: 1), ``norm.eps`` and
``layers``, a list whose entries give ``type``, ``mixer`` and ``mlp`` (``{"kind": "dense", "ff"}`` or null).  ``type``
"attention": ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size``, ``rot.dims``, ``rot.base``,
``v_mix``.  ``type`` "parallel": ``left`` (the same keys, without ``v_mix``), ``right`` (``heads``, ``dim``, ``vdim``,
``rot``, ``decay``: one number per head), ``left_scale``, ``right_scale``.  Every size and constant is read by key,
with an error that names the key; nothing is assumed equal between layers.  What a layer leaves out does not exist for
it: no ``mask``, every earlier token; no ``rot``, no rotation.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, _get
from .divanex import _obj, _sub

MIXERS = ("attention", "parallel")


@dataclass(frozen=True)
class Rotation:
    dims: int                    # how many of a head's first numbers are turned (0: none)
    base: float


@dataclass(frozen=True)
class SoftmaxAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]        # a query sees itself and the window - 1 tokens before it; None: all of them
    rot: Rotation
    v_mix: bool                  # the values are mixed with those of the first layer that says so


@dataclass(frozen=True)
class RetentionMixer:
    heads: int
    dim: int
    vdim: int
    rot: Rotation
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class ParallelMixer:
    left: SoftmaxAttention
    right: RetentionMixer
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class RanilixLayer:
    type: str
    mixer: Any                   # SoftmaxAttention | ParallelMixer
    ff: Optional[int]            # the feed-forward's inner width; None: no feed-forward


def _rotation(m: Dict[str, Any], dim: int, where: str) -> Rotation:
    rot = _obj(m, "rot", where, nullable=True)
    if rot is None:
        return Rotation(0, 1.0)
    r = Rotation(_sub(rot, "dims", int, where + "rot.", dim), _sub(rot, "base", float, where + "rot."))
    if r.dims % 2 or not 0 <= r.dims <= dim:
        raise ConfigError(f"config.json: {where}rot.dims={r.dims} must be even and at most dim={dim}")
    if not r.base > 0.0:
        raise ConfigError(f"config.json: {where}rot.base={r.base} must be positive")
    return r


def _attention(m: Dict[str, Any], where: str, mixes: bool) -> SoftmaxAttention:
    heads = _sub(m, "heads", int, where)
    dim = _sub(m, "dim", int, where)
    mask = _obj(m, "mask", where, nullable=True)
    v_mix = m.get("v_mix", False)
    if not isinstance(v_mix, bool) or (v_mix and not mixes):
        raise ConfigError(f"config.json: {where}v_mix={v_mix!r} must be true or false" + ("" if mixes else ", and false here"))
    a = SoftmaxAttention(heads, _sub(m, "kv_heads", int, where, heads), dim, _sub(m, "vdim", int, where, dim),
                         _sub(m, "scale", float, where), _sub(mask, "size", int, where + "mask.") if mask else None,
                         _rotation(m, dim, where), v_mix)
    if min(a.heads, a.kv_heads, a.dim, a.vdim) < 1 or a.heads % a.kv_heads:
        raise ConfigError(f"config.json: {where}heads, kv_heads, dim and vdim must be positive and kv_heads divide heads")
    if a.window is not None and a.window < 1:
        raise ConfigError(f"config.json: {where}mask.size={a.window} must be positive")
    return a


def _retention(m: Dict[str, Any], where: str) -> RetentionMixer:
    heads = _sub(m, "heads", int, where)
    dim = _sub(m, "dim", int, where)
    decay = m.get("decay")
    if not isinstance(decay, list) or any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay):
        raise ConfigError(f"config.json: {where}decay must be a list of numbers, got {decay!r}")
    r = RetentionMixer(heads, dim, _sub(m, "vdim", int, where, dim), _rotation(m, dim, where), tuple(float(x) for x in decay))
    if min(r.heads, r.dim, r.vdim) < 1:
        raise ConfigError(f"config.json: {where}heads, dim and vdim must be positive")
    if len(r.decay) != heads:
        raise ConfigError(f"config.json: {where}decay has {len(r.decay)} numbers for {heads} heads")
    return r


@dataclass(frozen=True)
class RanilixConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    layers: Tuple[RanilixLayer, ...]

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "RanilixConfig":
        vocab = _get(d, "vocab", int)
        width = _get(d, "width", int)
        if vocab < 1 or width < 1:
            raise ConfigError(f"config.json: vocab={vocab} and width={width} must be positive")
        norm = _obj(d, "norm", "")
        emb = _obj(d, "embedding", "", nullable=True) or {}
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers = []
        first = None                                     # the first layer whose values are mixed in: (index, mixer)
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            typ = _sub(L, "type", str, where)
            m = _obj(L, "mixer", where)
            if typ == "attention":
                mixer = _attention(m, where + "mixer.", True)
                if mixer.v_mix and first is None:
                    first = (i, mixer)
                elif mixer.v_mix and (mixer.kv_heads, mixer.vdim) != (first[1].kv_heads, first[1].vdim):
                    raise ConfigError(f"config.json: {where}mixer: {mixer.kv_heads} value heads of {mixer.vdim} cannot be mixed with "
                                      f"the {first[1].kv_heads} of {first[1].vdim} of layers[{first[0]}]")
            elif typ == "parallel":
                mixer = ParallelMixer(_attention(_obj(m, "left", where + "mixer."), where + "mixer.left.", False),
                                      _retention(_obj(m, "right", where + "mixer."), where + "mixer.right."),
                                      _sub(m, "left_scale", float, where + "mixer."), _sub(m, "right_scale", float, where + "mixer."))
            else:
                raise ConfigError(f"config.json: {where}type is '{typ}'; known mixers: {', '.join(MIXERS)}")
            ff = None
            ml = _obj(L, "mlp", where, nullable=True)
            if ml is not None:
                kind = _sub(ml, "kind", str, where + "mlp.")
                if kind != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind is '{kind}'; known kinds: dense")
                ff = _sub(ml, "ff", int, where + "mlp.")
                if ff < 1:
                    raise ConfigError(f"config.json: {where}mlp.ff={ff} must be positive")
            layers.append(RanilixLayer(typ, mixer, ff))
        return cls(vocab=vocab, width=width, embedding_scale=_sub(emb, "scale", float, "embedding.", 1.0),
                   norm_eps=_sub(norm, "eps", float, "norm."), layers=tuple(layers))
