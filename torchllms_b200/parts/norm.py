"""Root-mean-square norm, fused with the residual sum that precedes it.

Reference: ``RMSNorm.forward`` (torchllms/models/networks.py:195-200) squares,
averages and rescales in float32, casts back to the activation dtype and then
multiplies by the weight.  Here the stream itself is float32, the pending
delta is added in float32, and the weight is applied before the single
rounding to the activation dtype; in float32 the two orders are the same
arithmetic.

In bfloat16, when the part that reads the rows feeds them to a matrix product
first (``deferred_ok``), the rows leave as ``bf16(h * weight)`` with their sums
of squares, and the scale ``rsqrt(mean(h^2) + eps)`` is applied to the product
(a product is linear in its input): the same number with one rounding moved.
That lets a pending product add itself to the stream and prepare these rows in
its own epilogue, so that no norm kernel stands between two products of a
decode step.  Prompt portions go through the norm kernel in the same deferred
form, so that one arithmetic holds however a request is cut.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..kernels.lazy import PendingProduct
from ..weights.loader import ExpectedTensor
from .base import BuildEnv, Norm, Residual, register_norm


@register_norm("rmsnorm")
class RMSNorm(Norm):
    graph_safe = True
    can_defer = True

    def __init__(self, env: BuildEnv, *, dim: int, eps: float, offset: float = 0.0, scalar: bool = False, groups: int = 1,
                 weight_scale: float = 1.0):
        """``offset``: what is added to the stored weight (1 for a weight that is kept around zero).
        ``scalar``: the stored weight is one number for all coordinates (a tensor without axes).
        ``groups``: the row is cut into so many equal runs of neighbouring coordinates, each divided by a root
        mean square of its own (one scale per row is not enough then, so nothing is deferred).
        ``weight_scale``: what the weight is multiplied by, in 32-bit (a norm on a sublayer's output whose result enters
        the stream multiplied by a constant)."""
        if groups < 1 or dim % groups:
            raise ValueError(f"a norm over {dim} coordinates cannot have {groups} equal groups")
        self.groups = int(groups)
        self.can_defer = self.groups == 1
        self.env = env
        self.scalar = bool(scalar)
        self.dim = int(dim)
        self.eps = float(eps)
        self.offset, self.weight_scale = float(offset), float(weight_scale)
        self.weight: Optional[torch.Tensor] = None

    def expected_tensors(self) -> Dict[str, ExpectedTensor]:
        return {"weight": ExpectedTensor(() if self.scalar else (self.dim,))}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        # Kept in 32-bit whatever the activation dtype: the kernel multiplies in 32-bit.
        w = tensors["weight"].to(device=self.env.device, dtype=torch.float32) + self.offset
        if self.weight_scale != 1.0:
            w = w * self.weight_scale
        self.weight = (w.reshape(1).expand(self.dim) if self.scalar else w).contiguous()

    def forward(self, residual: Residual, rows: Optional[torch.Tensor] = None, deferred_ok: bool = False):
        ops = self.env.ops
        # 32-bit mode keeps the reference's order of operations to the letter
        deferred = bool(deferred_ok and rows is None and self.env.dtype == torch.bfloat16)
        delta, scale = residual.delta, residual.delta_scale
        if self.groups > 1 or scale is not None:
            out = ops.rmsnorm(residual.h, delta, self.weight, self.eps, out_dtype=self.env.dtype, rows=rows, groups=self.groups,
                              delta_scale=scale)
            if rows is None:
                residual.delta = residual.delta_scale = residual.rows = None
            return out
        if deferred and isinstance(delta, PendingProduct) and ops.can_fuse_residual(delta, residual.h):
            out = ops.linear_residual_norm(delta, residual.h, self.weight, self.eps)   # h += product, in the product's kernel
            residual.delta = None
            residual.rows = None
            return out
        if deferred:
            out = ops.rmsnorm(residual.h, delta, self.weight, self.eps, out_dtype=self.env.dtype, deferred=True)
        else:
            out = ops.rmsnorm(residual.h, delta, self.weight, self.eps, out_dtype=self.env.dtype, rows=rows)
        if rows is None:
            residual.delta = None  # the kernel wrote h + delta back into the stream
            residual.rows = None
        return out

    def fold_normed(self, residual: Residual, delta, want_rows: bool = True, then: Optional["RMSNorm"] = None):
        """The norm on a sublayer's *output*: ``h += norm(delta)`` in 32-bit, in one kernel that also
        leaves the new stream in the activation dtype (``residual.rows``) for the sublayer that
        reads it next (not with ``want_rows=False``: a reader that has a norm of its own in front).
        ``delta`` is a tensor, float32 partial sums or a
        :class:`~torchllms_b200.kernels.lazy.PendingProduct`.  With ``then`` (the norm in front of
        the next reader) the same kernel also returns ``then(h)`` in the activation dtype."""
        ops = self.env.ops
        if self.groups > 1 or (then is not None and then.groups > 1):
            raise RuntimeError("a norm with groups stands in front of a sublayer, not on its output")
        residual.delta = None
        if then is not None:
            residual.rows = None
            return ops.norm_add(residual.h, delta, self.weight, self.eps, out_dtype=self.env.dtype,
                                then_weight=then.weight, then_eps=then.eps)
        if not want_rows:
            ops.norm_add(residual.h, delta, self.weight, self.eps, out_dtype=torch.float32)
            residual.rows = None
            return None
        residual.rows = ops.norm_add(residual.h, delta, self.weight, self.eps, out_dtype=self.env.dtype)
        return None
