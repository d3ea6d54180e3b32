"""RMSNorm and layer norm, fused with the residual addition that precedes them.

out = x / sqrt(mean(x^2) + eps) * w with x = residual (+ delta); reduced in
float32.  src/model/math.rs:28-50.
"""
from __future__ import annotations

from typing import List

from ..config.spec import NormSpec
from ..kernels import ops
from ..weights.loader import VECTOR, TensorDecl
from .base import Part, register_norm, split_delta


@register_norm("rmsnorm")
class RMSNorm(Part):
    center = False

    def __init__(self, spec: NormSpec, name: str, tensors: dict, mctx):
        self.spec, self.weight = spec, tensors[name]

    @classmethod
    def tensor_decls(cls, spec: NormSpec, name: str) -> List[TensorDecl]:
        return [TensorDecl(name, (spec.size,), VECTOR)]

    @property
    def fusable(self) -> bool:
        """Whether products may apply this norm in their own prologue and epilogue (parts.base.NormedInput)."""
        return not self.spec.unit_offset

    def apply(self, residual, delta, out, rows=None):
        """residual[float32] += delta (kept when rows is None; a ScaledDelta: times its scale); out = norm of the sum.
        With ``rows`` only those rows are normed, into out[0..len(rows))."""
        delta, scale = split_delta(delta)
        ops.add_norm(residual, delta, self.weight, self.spec.eps, out, rows, self.spec.unit_offset, self.center, scale)


@register_norm("layernorm")
class LayerNorm(RMSNorm):
    """Layer norm with a weight and no bias: out = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w."""
    center = True
    fusable = False        # the products' prologues and epilogues form sums of squares, not deviations from a mean


@register_norm("rmsnorm_scalar")
class ScalarRMSNorm(RMSNorm):
    """RMSNorm whose scale is one number for all coordinates, stored as a tensor of shape ().  The number
    is repeated over the width once, when the part is built, and the kernels of the vector norm serve."""
    fusable = False        # the products' norm prologues and epilogues are not offered to blocks that use this norm

    def __init__(self, spec: NormSpec, name: str, tensors: dict, mctx):
        self.spec = spec
        self.weight = tensors[name].reshape(1).expand(spec.size).contiguous()

    @classmethod
    def tensor_decls(cls, spec: NormSpec, name: str) -> List[TensorDecl]:
        return [TensorDecl(name, (), VECTOR)]
