"""Sezanex as data: its configuration turned into a :class:`ModelSpec`.

Nothing here computes.  A Sezanex layer is a ``sandwich`` block, a norm before and a norm after each sublayer, all of
them dynamic tanh norms (:class:`trapetum_b200.parts.norm.DynamicTanh`), around one of two mixers and a feed-forward:

* ``attention`` is :mod:`trapetum_b200.parts.attention` with q and k RMS-normed over the whole projection, a rotation of
  the first ``rot.dims`` numbers of every head with frequencies blended between their own and the scaled ones, a sliding
  window, values of their own size, and a softmax with one added to its denominator;
* ``mamba2`` is :mod:`trapetum_b200.parts.mamba2`;
* the feed-forward is ``down(gelu(up x))`` with the exact gelu, or :mod:`trapetum_b200.parts.experts`: gated experts with
  silu behind sigmoid scores, which are neither renormalised nor applied to the expert's output but to its input.

A span of layers may run several times in a row with the same weights: the schedule names those layers once per pass,
every call owns a cache of its own, and the first call of a pass carries a ``project_input`` that replaces the stream by
a product of itself beside the embedding's output.  The head multiplies with the embedding table.

Tensor names: ``embed``, ``loop.in``, ``l<i>.norm{1,1b,2,2b}`` (each with ``.b`` and ``.alpha``), ``l<i>.mix.{q,k,v,o}``,
``l<i>.mix.{q,k}.norm``, ``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``, ``l<i>.mlp.{up,down}``, ``l<i>.mlp.router``,
``l<i>.mlp.e<j>.{gate,up,down}``, ``final.norm`` (with ``.b`` and ``.alpha``).
"""
from __future__ import annotations

from ..config.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, register_architecture
from ..config.sezanex import PlainMlp, SezanexConfig

MAX_POSITIONS = 1 << 24          # angles are position x frequency in 32-bit: every integer up to here is exact


def sezanex_spec(cfg: SezanexConfig) -> ModelSpec:
    W = cfg.width

    def norm(name: str) -> PartSpec:
        return PartSpec("dynamic_tanh", {"size": W, "weight": name, "bias": name + ".b", "alpha": name + ".alpha"})

    layers = []
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        if L.type == "attention":
            position = PartSpec("none", {"head_dim": m.dim})
            if m.rot.dims:
                position = PartSpec("rope", {"head_dim": m.dim, "rotary_dim": m.rot.dims, "theta": m.rot.base,
                                             "scaling": m.rot.scaling, "table": "float64"})
            mixer = PartSpec("attention", {
                "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
                "scale": m.scale, "softcap": None, "window": m.window, "unit_sink": True, "position": position,
                "proj_norm": {"q": "mix.q.norm", "k": "mix.k.norm", "eps": cfg.norm_eps},
                "q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o",
            })
        else:
            mixer = PartSpec("mamba2", {
                "hidden_size": W, "heads": m.heads, "head_dim": m.vdim, "state": m.state, "groups": m.groups,
                "conv": m.conv, "norm_groups": m.norm_groups, "eps": cfg.norm_eps,
                "in": "mix.in", "conv_w": "mix.conv", "conv_b": "mix.conv.b", "dt_bias": "mix.dt_bias",
                "A_log": "mix.A_log", "D": "mix.D", "norm": "mix.norm", "o": "mix.o",
            })
        if L.mlp is None:
            ffn = PartSpec("none", {})
        elif isinstance(L.mlp, PlainMlp):
            ffn = PartSpec("mlp", {"hidden_size": W, "intermediate_size": L.mlp.ff, "activation": "gelu",
                                   "up": "mlp.up", "down": "mlp.down"})
        else:
            ffn = PartSpec("routed_experts", {
                "hidden_size": W, "experts": L.mlp.experts, "top": L.mlp.top, "intermediate_size": L.mlp.ff,
                "activation": "silu", "score": "sigmoid", "renormalize": False, "weight_on": "input",
                "router": "mlp.router", "correction": None,
                "expert": "mlp.e{}.", "gate": "gate", "up": "up", "down": "down", "shared": None,
            })
        params = {"pre_mixer_norm": norm("norm1"), "post_mixer_norm": norm("norm1b"),
                  "pre_ffn_norm": None, "post_ffn_norm": None}
        if L.mlp is not None:
            params.update(pre_ffn_norm=norm("norm2"), post_ffn_norm=norm("norm2b"))
        else:
            params["idle"] = {n + end: shape for n in ("norm2", "norm2b") for end, shape in (("", W), (".b", W), (".alpha", []))}
        layers.append(LayerSpec(block=PartSpec("sandwich", params), mixer=mixer, feed_forward=ffn, prefix=f"l{i}."))

    n = len(layers)
    schedule = [ScheduleEntry(i) for i in range(n)]
    if cfg.loop is not None:
        lp = cfg.loop
        before = PartSpec("project_input", {"hidden_size": W, "weight": "loop.in"})
        one_pass = [ScheduleEntry(i, before=before if i == lp.start else None) for i in range(lp.start, lp.stop)]
        schedule = schedule[:lp.start] + one_pass * lp.times + schedule[lp.stop:]

    return ModelSpec(
        architecture="Sezanex",
        hidden_size=W,
        vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "scale": 1.0, "weight": "embed"}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "softcap": None, "scale": None,
                                      "weight": "embed", "tied_to": None}),
        max_positions=MAX_POSITIONS,
        stop_ids=(),
    )


register_architecture("Sezanex", SezanexConfig, sezanex_spec, native=False)
