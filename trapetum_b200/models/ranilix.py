"""Ranilix as data: its configuration turned into a :class:`ModelSpec`.

Nothing here computes.  A Ranilix layer is a ``parallel`` block with two norms: the mixer and the feed-forward read the
same stream, each through an RMS norm of its own, and their outputs are added to it together.  Two mixers:

* "attention" is :mod:`trapetum_b200.parts.attention` with biases, q and k RMS-normed per head, a rotation of neighbouring
  pairs over the first ``rot.dims`` numbers of a head, a sliding window, a sink per head in the softmax denominator,
  values mixed with the first such layer's, values of their own size, and a sigmoid gate on every output number;
* "parallel" is :mod:`trapetum_b200.parts.side_by_side`: attention without any of these but the rotation and values of
  their own size, beside :mod:`trapetum_b200.parts.retention` (a rotation of halves), added with a scale each.

The feed-forward is ``down(relu(up x)^2)``.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.{q,k,v}``, ``l<i>.mix.{q,k,v}.b``,
``l<i>.mix.{q,k}.norm``, ``l<i>.mix.{vmix,sink,g,o}``, ``l<i>.mix.left.{q,k,v,o}``, ``l<i>.mix.right.{q,k,v,g,o}``,
``l<i>.mlp.{up,down}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, register_architecture
from ..config.ranilix import RanilixConfig

MAX_POSITIONS = 1 << 24          # angles are position x frequency in 32-bit: every integer up to here is exact


def _position(rot, dim: int, pairing: str) -> PartSpec:
    if not rot.dims:
        return PartSpec("none", {"head_dim": dim})
    return PartSpec("rope", {"head_dim": dim, "rotary_dim": rot.dims, "theta": rot.base, "pairing": pairing, "table": "float64"})


def _attention(m, width: int, at: str, extra: dict) -> PartSpec:
    params = {"hidden_size": width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
              "scale": m.scale, "softcap": None, "window": m.window, "position": _position(m.rot, m.dim, "neighbours"),
              "q": at + "q", "k": at + "k", "v": at + "v", "o": at + "o"}
    params.update(extra)
    return PartSpec("attention", params)


def ranilix_spec(cfg: RanilixConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": eps, "weight": name, "role": "gain"})

    layers, mixed = [], False
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        if L.type == "attention":
            extra = {"bias": {"q": "mix.q.b", "k": "mix.k.b", "v": "mix.v.b"},
                     "head_norm": {"q": "mix.q.norm", "k": "mix.k.norm", "eps": eps},
                     "sink": "mix.sink", "value_gate": "mix.g"}
            if m.v_mix:
                extra["v_mix"] = {"weight": "mix.vmix", "first": not mixed, "group": "v"}
                mixed = True
            mixer = _attention(m, W, "mix.", extra)
        else:
            r = m.right
            mixer = PartSpec("side_by_side", {
                "left": _attention(m.left, W, "mix.left.", {}),
                "right": PartSpec("retention", {
                    "hidden_size": W, "heads": r.heads, "key_dim": r.dim, "value_dim": r.vdim, "decay": list(r.decay),
                    "k_scale": None, "eps": eps, "position": _position(r.rot, r.dim, "halves"),
                    "q": "mix.right.q", "k": "mix.right.k", "v": "mix.right.v", "g": "mix.right.g", "o": "mix.right.o"}),
                "left_scale": m.left_scale, "right_scale": m.right_scale})
        if L.ff is not None:
            ffn = PartSpec("mlp", {"hidden_size": W, "intermediate_size": L.ff, "activation": "relu2",
                                   "up": "mlp.up", "down": "mlp.down"})
            block = PartSpec("parallel", {"norm": norm("norm1"), "ffn_norm": norm("norm2")})
        else:
            ffn = PartSpec("none", {})
            block = PartSpec("parallel", {"norm": norm("norm1"), "idle": {"norm2": W}})
        layers.append(LayerSpec(block=block, mixer=mixer, feed_forward=ffn, prefix=f"l{i}."))

    return ModelSpec(
        architecture="Ranilix",
        hidden_size=W,
        vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "scale": cfg.embedding_scale, "weight": "embed"}),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "softcap": None, "scale": None,
                                      "weight": "head", "tied_to": None}),
        max_positions=MAX_POSITIONS,
        stop_ids=(),
    )


register_architecture("Ranilix", RanilixConfig, ranilix_spec, native=False)
