"""Two mixers side by side: both read the same rows, and the result is a weighted sum of their
outputs, either each RMS-normed over the stream's width first (``side_by_side``) or as they are
(``side_by_side_sum``).

One of the two may keep keys and values in the paged cache and either may keep state rows; the
pair asks the cache manager for both in its members' names and hands each member what is its own.
"""

from __future__ import annotations

import dataclasses
from typing import Dict, Mapping, Optional

import torch

from ..kernels.lazy import NormedSum, PendingProduct
from ..weights.loader import ExpectedTensor
from .base import MIXERS, BuildEnv, Mixer, join_states, register_mixer, state_field
from .spec import PartSpec


class _Pair(Mixer):
    """What any two mixers side by side have in common: the members, and what they want of the cache manager."""

    def __init__(self, env: BuildEnv, left: PartSpec, right: PartSpec, left_prefix: str, right_prefix: str):
        self.env = env
        self.members = ((left_prefix, MIXERS.build(left, env)), (right_prefix, MIXERS.build(right, env)))
        if sum(m.cache_need() is not None for _p, m in self.members) > 1:
            raise ValueError("of two mixers side by side at most one may keep keys and values in the paged cache")
        self.graph_safe = all(m.graph_safe for _p, m in self.members)
        self._need = join_states([(p, m.state_need()) for p, m in self.members])

    def cache_need(self):
        for _p, m in self.members:
            if m.cache_need() is not None:
                return m.cache_need()
        return None

    def state_need(self):
        return self._need

    def expected_tensors(self) -> Dict[str, ExpectedTensor]:
        return {f"{prefix}.{name}": e for prefix, m in self.members for name, e in m.expected_tensors().items()}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for prefix, m in self.members:
            m.load({name: tensors[f"{prefix}.{name}"] for name in m.expected_tensors()})

    def _cache_of(self, prefix: str, m: Mixer, cache):
        state = None if m.state_need() is None else state_field(cache.state, self._need, prefix)
        return dataclasses.replace(cache, state=state)


@register_mixer("side_by_side")
class SideBySide(_Pair):
    """``coef * (norm_l(left(x)) + norm_r(right(x)))`` with plain-weight RMS norms over the width.

    Tensors: the members' under ``<left_prefix>.`` and ``<right_prefix>.``, the norms' weights
    ``<left_prefix>.<out_norm>`` and ``<right_prefix>.<out_norm>``.  The sum is left untaken
    (:class:`~torchllms_b200.kernels.lazy.NormedSum`): the kernel that adds the layer's result to
    the stream takes both norms in 32-bit on the way."""

    def __init__(self, env: BuildEnv, *, dim: int, left: PartSpec, right: PartSpec, eps: float, coef: float = 0.5,
                 left_prefix: str = "left", right_prefix: str = "right", out_norm: str = "out"):
        super().__init__(env, left, right, left_prefix, right_prefix)
        self.dim, self.eps, self.coef, self.out_norm = int(dim), float(eps), float(coef), out_norm
        self.out_w: Dict[str, torch.Tensor] = {}

    def expected_tensors(self) -> Dict[str, ExpectedTensor]:
        out = super().expected_tensors()
        for prefix, _m in self.members:
            out[f"{prefix}.{self.out_norm}"] = ExpectedTensor((self.dim,))
        return out

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        super().load(tensors)
        for prefix, _m in self.members:
            self.out_w[prefix] = tensors[f"{prefix}.{self.out_norm}"].to(device=self.env.device, dtype=torch.float32).contiguous()

    def weight_bytes(self) -> int:
        return sum(m.weight_bytes() for _p, m in self.members)

    def forward(self, x: torch.Tensor, ctx, cache) -> NormedSum:
        terms = []
        for prefix, m in self.members:
            y = m.forward(x, ctx, self._cache_of(prefix, m, cache))
            if isinstance(y, PendingProduct):
                y = y.take(self.env.ops, partials_ok=True)
            terms.append((y, self.out_w[prefix]))
        return NormedSum(tuple(terms), self.coef, self.eps)


@register_mixer("side_by_side_sum")
class SideBySideSum(_Pair):
    """``left(x) + right(x)``, each member scaled by what its own ``out_scale`` says, for members that run in halves
    (``Mixer.runs_in_halves``): their input products are one product over the stacked weights, each writes its result
    into its columns of one row, and ``[left's rows | right's rows]`` times ``[wo_l | wo_r]`` is the sum: one product, left to
    the norm that follows.  Between the two products the members of a step of short portions run on two streams."""

    def __init__(self, env: BuildEnv, *, dim: int, left: PartSpec, right: PartSpec, left_prefix: str = "left",
                 right_prefix: str = "right"):
        super().__init__(env, left, right, left_prefix, right_prefix)
        self.dim = int(dim)
        for prefix, m in self.members:
            if not m.runs_in_halves:
                raise ValueError(f"the {prefix} mixer of a sum of two does not run in halves")
        self.widths = self.inner = ()
        self.w_in: Optional[torch.Tensor] = None
        self.wo: Optional[torch.Tensor] = None

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        super().load(tensors)
        parts = [m for _p, m in self.members]
        self.widths, self.inner = tuple(m.w_in.shape[0] for m in parts), tuple(m.wo.shape[1] for m in parts)
        self.w_in = torch.cat([m.w_in for m in parts]).contiguous()
        self.wo = torch.cat([m.wo for m in parts], dim=1).contiguous()
        for m in parts:
            m.w_in = m.wo = None                      # the stacked weights stand in for the members' own

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.wo)) + sum(m.weight_bytes() for _p, m in self.members)

    def forward(self, x: torch.Tensor, ctx, cache) -> PendingProduct:
        proj = self.env.ops.linear(x, self.w_in, partials_ok=True)
        rows = torch.empty((x.shape[0], sum(self.inner)), dtype=self.env.dtype, device=x.device)
        at, to = self.widths[0], self.inner[0]
        (lp, left), (rp, right) = self.members
        # the members know nothing of each other: their kernels may run side by side
        with self.env.ops.aside(ctx.max_q_len):
            right.mix(proj[..., at:], ctx, self._cache_of(rp, right, cache), rows[:, to:])
        left.mix(proj[..., :at], ctx, self._cache_of(lp, left, cache), rows[:, :to])
        self.env.ops.rejoin()
        return PendingProduct(rows, self.wo)
