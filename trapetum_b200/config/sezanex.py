"""Sezanex's configuration, read from the keys of its config.json.

Top level: ``architecture`` ("Sezanex"), ``vocab``, ``width``, ``norm.eps``, ``loop`` (``start``, ``stop``, ``times``;
absent: every layer runs once) and ``layers``, a list whose entries give ``type`` (one of the mixers below), ``mixer``
(its sizes and constants) and ``mlp`` (``{"kind": "dense", "ff"}``, ``{"kind": "moe", "expert": {"ff"}, "router":
{"experts", "top"}}`` or null).

``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (a sliding window), ``rot.dims``,
``rot.base``, ``rot.scaling`` (``factor``, ``original``, ``fast``, ``slow``: a blend per frequency).
``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv``, ``norm_groups``.

Every size and constant is read by key, with an error that names the key; nothing is assumed equal between layers.
What a layer leaves out does not exist for it: no ``mask``, every earlier token is seen; no ``rot``, no rotation; no
``scaling``, frequencies as they are; ``mlp`` null, no feed-forward.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, _get
from .divanex import Mamba2Mixer, _obj, _sub
from .fibelix import Rotation, TopMoe, _mask, _rotation
from .lofirax import Loop

MIXERS = ("attention", "mamba2")


@dataclass(frozen=True)
class SinkAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]        # a query sees itself and the window - 1 tokens before it; None: all of them
    rot: Rotation


@dataclass(frozen=True)
class PlainMlp:
    ff: int


@dataclass(frozen=True)
class SezanexLayer:
    type: str
    mixer: Any                   # SinkAttention | Mamba2Mixer
    mlp: Any                     # PlainMlp | TopMoe | None


def _attention(m, mw) -> SinkAttention:
    heads = _sub(m, "heads", int, mw)
    kv_heads = _sub(m, "kv_heads", int, mw, heads)
    dim = _sub(m, "dim", int, mw)
    vdim = _sub(m, "vdim", int, mw, dim)
    if min(heads, kv_heads, dim, vdim) < 1 or heads % kv_heads:
        raise ConfigError(f"config.json: {mw}heads={heads}, kv_heads={kv_heads}, dim={dim} and vdim={vdim} must be positive, "
                          "kv_heads a divisor of heads")
    return SinkAttention(heads, kv_heads, dim, vdim, _sub(m, "scale", float, mw), _mask(m, mw), _rotation(m, mw, dim))


def _mamba2(m, mw) -> Mamba2Mixer:
    mixer = Mamba2Mixer(*(_sub(m, key, int, mw) for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
    if min(mixer.heads, mixer.vdim, mixer.state, mixer.groups, mixer.conv, mixer.norm_groups) < 1:
        raise ConfigError(f"config.json: {mw}heads, vdim, state, groups, conv and norm_groups must be positive")
    if mixer.heads % mixer.groups or (mixer.heads * mixer.vdim) % mixer.norm_groups:
        raise ConfigError(f"config.json: {mw}groups={mixer.groups} must divide heads={mixer.heads}, and "
                          f"norm_groups={mixer.norm_groups} must divide heads * vdim = {mixer.heads * mixer.vdim}")
    return mixer


def _mlp(ml, lw):
    kind = _sub(ml, "kind", str, lw)
    if kind == "dense":
        mlp = PlainMlp(_sub(ml, "ff", int, lw))
        if mlp.ff < 1:
            raise ConfigError(f"config.json: {lw}ff={mlp.ff} must be positive")
        return mlp
    if kind != "moe":
        raise ConfigError(f"config.json: {lw}kind is '{kind}'; known kinds: dense, moe")
    r = _obj(ml, "router", lw)
    mlp = TopMoe(_sub(r, "experts", int, lw + "router."), _sub(r, "top", int, lw + "router."),
                 _sub(_obj(ml, "expert", lw), "ff", int, lw + "expert."))
    if mlp.experts < 1 or mlp.ff < 1 or not (1 <= mlp.top <= mlp.experts):
        raise ConfigError(f"config.json: {lw}router: top={mlp.top} of experts={mlp.experts}, ff={mlp.ff}")
    return mlp


@dataclass(frozen=True)
class SezanexConfig:
    vocab: int
    width: int
    norm_eps: float
    loop: Optional[Loop]
    layers: Tuple[SezanexLayer, ...]

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "SezanexConfig":
        vocab = _get(d, "vocab", int)
        width = _get(d, "width", int)
        if vocab < 1 or width < 1:
            raise ConfigError(f"config.json: vocab={vocab} and width={width} must be positive")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            typ = _sub(L, "type", str, where)
            if typ not in MIXERS:
                raise ConfigError(f"config.json: {where}type is '{typ}'; known mixers: {', '.join(MIXERS)}")
            read = _attention if typ == "attention" else _mamba2
            mixer = read(_obj(L, "mixer", where), where + "mixer.")
            ml = _obj(L, "mlp", where, nullable=True)
            layers.append(SezanexLayer(typ, mixer, None if ml is None else _mlp(ml, where + "mlp.")))
        loop = None
        lp = _obj(d, "loop", "", nullable=True)
        if lp is not None:
            loop = Loop(_sub(lp, "start", int, "loop."), _sub(lp, "stop", int, "loop."), _sub(lp, "times", int, "loop."))
            if not (0 <= loop.start < loop.stop <= len(layers)) or loop.times < 1:
                raise ConfigError(f"config.json: loop start={loop.start} stop={loop.stop} times={loop.times} does not "
                                  f"fit {len(layers)} layers")
        return cls(vocab=vocab, width=width, norm_eps=_sub(_obj(d, "norm", ""), "eps", float, "norm."), loop=loop,
                   layers=tuple(layers))
