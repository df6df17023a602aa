"""Two mixers side by side: both read the same input, and their outputs are added with a scale each.

``left_scale * left(h) + right_scale * right(h)``.  Parameters: ``left`` and ``right`` (mixer specs; their tensor names
are their own), ``left_scale``, ``right_scale``.  At most one of the two may keep keys and values and at most one a
state; the cache then holds both for the one schedule entry.  When both can finish from their input product
(``in_weight``, ``finish``), the two input matrices are one product.  The scaled sum is left to the block
(:class:`~trapetum_b200.parts.base.Terms`).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..weights.loader import TensorSpec
from .base import KVNeed, Mixer, StateNeed, Terms, build_part, register_part
from .linear import linear_partials


class SideBySide(Mixer):
    def __init__(self, params, prefix, rt):
        super().__init__(params, prefix, rt)
        self.left = build_part("mixer", params["left"], prefix, rt)
        self.right = build_part("mixer", params["right"], prefix, rt)
        self.scales = (float(params["left_scale"]), float(params["right_scale"]))
        self.needs = [m.cache_need() for m in (self.left, self.right)]
        for kind in (KVNeed, StateNeed):
            if sum(isinstance(n, kind) for n in self.needs) > 1:
                raise ValueError(f"side_by_side: both mixers ask for a {kind.__name__}; one schedule entry holds one of each")
        if any(isinstance(n, tuple) for n in self.needs):
            raise ValueError("side_by_side: a side that itself keeps both keys and a state is not built")
        self.w_in = None

    @property
    def graph_safe(self):
        return all(getattr(m, "graph_safe", False) for m in (self.left, self.right))

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {**self.left.tensor_specs(), **self.right.tensor_specs()}

    def bind(self, tensors) -> None:
        self.left.bind(tensors)
        self.right.bind(tensors)
        if all(hasattr(m, "finish") for m in (self.left, self.right)):
            a, b = self.left.in_weight, self.right.in_weight
            if a.dtype == b.dtype:
                # the right side's columns begin on a whole tile of weight rows
                gap = torch.zeros((-a.shape[0] % 16, a.shape[1]), dtype=a.dtype, device=a.device)
                self.right_col = a.shape[0] + gap.shape[0]
                self.w_in = torch.cat([a, gap, b], dim=0).contiguous()
                # one copy of the weights: the sides' matrices become views of it
                self.left.in_weight = self.w_in[:a.shape[0]]
                self.right.in_weight = self.w_in[self.right_col:]

    def kernel_files(self):
        return tuple(self.left.kernel_files()) + tuple(self.right.kernel_files())

    def cache_need(self):
        have = [n for n in self.needs if n is not None]
        return None if not have else have[0] if len(have) == 1 else tuple(have)

    def _views(self, cache):
        """The cache as each side sees it."""
        if all(n is not None for n in self.needs):
            return tuple(cache.kv if isinstance(n, KVNeed) else cache.state for n in self.needs)
        return tuple(cache if n is not None else None for n in self.needs)

    def forward(self, x, ctx, cache):
        lc, rc = self._views(cache)
        if self.w_in is not None:
            part = linear_partials(x, self.w_in)
            a = self.left.finish(part[:, :, :self.right_col], ctx, lc)
            b = self.right.finish(part[:, :, self.right_col:], ctx, rc)
        else:
            a, b = self.left.forward(x, ctx, lc), self.right.forward(x, ctx, rc)
        return Terms(((a, self.scales[0]), (b, self.scales[1])))


register_part("mixer", "side_by_side", SideBySide)
