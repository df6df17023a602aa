"""Retention: a recurrent mixer whose state is a matrix per head that decays by a constant of the head.

Between a fused input product ``[q | k | v | g] = W h`` and an output product ``W_o``, per head (key channels d, value
channels v):

* q and k are turned at the token's position (``position``: a rotation of halves or of neighbours, or none), k is
  multiplied by ``k_scale`` (None: ``key_dim ** -0.5``);
* ``S <- decay S + k_t v_t^T`` and ``o_t = S^T q_t``, with no softmax and no denominator;
* every head's ``o_t`` is divided by its root mean square (eps inside the root, no weight) and multiplied by
  ``silu(g_t)``.

A sequence's state ``[heads, key_dim, value_dim]`` is one float32 row of the cache's state area, addressed by slot,
zero when the sequence starts, carried from step to step.  32-bit: angles, the turned q and k, the decay, the state,
``o``, its norm and the gate; v is rounded to the compute dtype.

Parameters (none is fixed in code): ``hidden_size``, ``heads``, ``key_dim``, ``value_dim``, ``decay`` (one number per
head), ``k_scale``, ``eps``, ``position`` and the tensor names ``q``, ``k``, ``v``, ``g``, ``o``.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from ..weights.loader import TensorSpec
from .base import Mixer, StateNeed, build_part, register_part
from .linear import kernel_files as linear_kernels
from .linear import linear_partials


class Retention(Mixer):
    graph_safe = True          # sequences, slots and positions are read on the device

    def __init__(self, params, prefix, rt):
        super().__init__(params, prefix, rt)
        p = params
        self.hidden = int(p["hidden_size"])
        self.heads = int(p["heads"])
        self.D = int(p["key_dim"])
        self.V = int(p["value_dim"])
        self.eps = float(p["eps"])
        self.k_scale = float(p["k_scale"]) if p.get("k_scale") is not None else self.D ** -0.5
        self.decays = [float(x) for x in p["decay"]]
        if min(self.heads, self.D, self.V) < 1 or len(self.decays) != self.heads:
            raise ValueError(f"retention: heads={self.heads} key_dim={self.D} value_dim={self.V} with {len(self.decays)} decays")
        self.position = build_part("position", p["position"], prefix, rt)
        if self.position.rotary_table() is None:
            raise ValueError("retention: 'position' must be a rotation or none")
        if self.position.amplitude != 1.0:
            raise ValueError("retention: a rotation with a factor on cos and sin is not built")

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        HD, HV = self.heads * self.D, self.heads * self.V
        return {self._name(key): TensorSpec(shape) for key, shape in (
            ("q", (HD, self.hidden)), ("k", (HD, self.hidden)), ("v", (HV, self.hidden)), ("g", (HV, self.hidden)),
            ("o", (self.hidden, HV)))}

    def bind(self, tensors) -> None:
        mats = [tensors[self._name(n)] for n in ("q", "k", "v", "g")]
        order = self.position.head_order()
        if order is not None:
            idx = torch.tensor(order, device=mats[0].device)
            mats[:2] = [m.view(self.heads, self.D, self.hidden)[:, idx].reshape(m.shape) for m in mats[:2]]
        dt = mats[0].dtype if all(m.dtype == mats[0].dtype for m in mats) else torch.float32
        n = sum(m.shape[0] for m in mats)
        mats.append(torch.zeros((-n % 16, self.hidden), dtype=dt, device=mats[0].device))        # whole tiles of weight rows
        self.w_in = torch.cat([m.to(dt) for m in mats], dim=0).contiguous()
        self.w_o = tensors[self._name("o")]
        self.decay = torch.tensor(self.decays, dtype=torch.float32, device=self.w_in.device)
        self.position.bind(tensors)

    def kernel_files(self):
        return linear_kernels(self.rt.dtype) + ops.retention_files(self.rt.dtype, self.D, self.V)

    def cache_need(self):
        return StateNeed((self.heads * self.D * self.V,), torch.float32)

    @property
    def in_weight(self) -> torch.Tensor:
        """The fused input matrix (see :meth:`finish`)."""
        return self.w_in

    @in_weight.setter
    def in_weight(self, w: torch.Tensor) -> None:
        self.w_in = w

    def finish(self, part, ctx, state):
        """The rest of the mixer: ``part`` is the product with ``in_weight`` as 32-bit partial sums [splits, T, width]."""
        inv_freq, rotary = self.position.rotary_table()
        y = ops.retention(part, self.heads, self.D, self.V, self.rt.dtype, rotary, inv_freq, self.k_scale, self.decay, self.eps,
                          state.data, ctx.positions, ctx.seq_start, ctx.token_seq, ctx.slot_ids, ctx.batch,
                          max_seq_len=ctx.max_seq_len if ctx.is_prefill else 0)
        return linear_partials(y, self.w_o)

    def forward(self, x, ctx, state):
        return self.finish(linear_partials(x, self.w_in), ctx, state)


register_part("mixer", "retention", Retention)
