"""Gated dense feed-forward: down(act(gate(x)) * up(x)), SiLU as the activation.
src/model/native.rs:552-557, src/model/math.rs:11-22."""
from __future__ import annotations

from typing import List

import torch

from ..config.spec import FeedForwardSpec
from ..errors import Unsupported
from ..kernels import ops
from ..weights.loader import MATRIX, TensorDecl
from .base import Part, register_feed_forward
from .linear import Linear


@register_feed_forward("gated_dense")
class GatedDense(Part):
    def __init__(self, spec: FeedForwardSpec, prefix: str, tensors: dict, mctx):
        if spec.activation != "silu":
            raise Unsupported(f"activation {spec.activation!r} is not implemented")
        self.spec = spec
        p, nm = prefix, spec.names
        gate, up = tensors[p + nm.gate], tensors[p + nm.up]
        I, H = gate.shape
        # One projection for gate and up.  For the tensor-core kernels the rows are interleaved in
        # blocks of 16 (8 gate rows, then the 8 up rows of the same features) so that the product's
        # epilogue holds both halves of a feature and writes silu(gate) * up directly; otherwise gate
        # rows then up rows, and a SwiGLU kernel halves the output.
        self.fused = (I % 8 == 0 and gate.dtype == torch.bfloat16 and mctx.dtype == torch.bfloat16
                      and H % 8 == 0 and not mctx.options.get("unfused_swiglu", False))
        if self.fused:
            w = torch.stack([gate.view(I // 8, 8, H), up.view(I // 8, 8, H)], dim=1).reshape(2 * I, H)
        else:
            w = torch.cat([gate, up], dim=0)
        self.gate_up = Linear(w.contiguous(), p + "gate_up")
        self.down = Linear(tensors[p + nm.down], p + nm.down)

    @classmethod
    def tensor_decls(cls, spec: FeedForwardSpec, prefix: str) -> List[TensorDecl]:
        p, nm = prefix, spec.names
        return [TensorDecl(p + nm.gate, (spec.intermediate_size, spec.hidden_size), MATRIX),
                TensorDecl(p + nm.up, (spec.intermediate_size, spec.hidden_size), MATRIX),
                TensorDecl(p + nm.down, (spec.hidden_size, spec.intermediate_size), MATRIX)]

    def can_fuse(self, ctx) -> bool:
        return self.fused and self.gate_up.can_fuse(ctx, ctx.T) and self.down.can_fuse(ctx, ctx.T)

    def forward_fused(self, ctx, nx, residual: torch.Tensor, next_norm):
        """forward for a lazily normalised input; the down projection adds into the residual stream and
        prepares the input of the part behind ``next_norm`` (None: nothing follows)."""
        h = ctx.workspace.get("ffn.h", ctx.T, self.spec.intermediate_size, ctx.dtype)
        self.gate_up.from_normed(ctx, nx, h, swiglu8=True)
        return self.down.into_residual(ctx, h, residual, next_norm, "f")

    def forward(self, ctx, x: torch.Tensor) -> torch.Tensor:
        h = ctx.workspace.get("ffn.h", x.shape[0], self.spec.intermediate_size, ctx.dtype)
        if self.fused and ops.can_fuse_swiglu(x.dtype, self.gate_up.weight):
            ops.gemm(x, self.gate_up.weight, h, swiglu8=True)
        else:
            gu = self.gate_up(ctx, x, "ffn.gate_up")
            ops.swiglu(gu, h)
        return self.down(ctx, h, "ffn.down")


@register_feed_forward("dense")
class Dense(Part):
    """down(act(up(x))) without a gate; ``activation`` "gelu": the exact one, "relu_squared": max(z, 0)^2.  The first
    product writes float32 and the activation rounds once, into the second product's input; in steps of many tokens the
    activation rides in the first product's epilogue (the grouped tensor-memory product with one group), where the sum is
    float32 too."""

    FUSED_TOKENS = 256       # least tokens of a step whose activation rides in the product

    def __init__(self, spec, prefix: str, tensors: dict, mctx):
        if spec.activation not in ("gelu", "relu_squared"):
            raise Unsupported(f"a dense feed-forward with activation {spec.activation!r} is not implemented")
        self.spec = spec
        nm = spec.dense_names
        self.up = Linear(tensors[prefix + nm.up], prefix + nm.up)
        w = self.up.weight
        self.fused = mctx.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0
        self.one_group = torch.zeros(-(-mctx.max_batch_tokens // ops.GROUPED_TILE) + 1, dtype=torch.int32, device=mctx.device)
        self.down = Linear(tensors[prefix + nm.down], prefix + nm.down)

    @classmethod
    def tensor_decls(cls, spec, prefix: str) -> List[TensorDecl]:
        nm = spec.dense_names
        return [TensorDecl(prefix + nm.up, (spec.intermediate_size, spec.hidden_size), MATRIX),
                TensorDecl(prefix + nm.down, (spec.hidden_size, spec.intermediate_size), MATRIX)]

    def forward(self, ctx, x: torch.Tensor) -> torch.Tensor:
        T, (I, H) = x.shape[0], self.up.weight.shape
        h = ctx.workspace.get("dense.h", T, I, ctx.dtype)
        tile = ops.grouped_tile_rows(T, 1, I * H)
        if (self.fused and ops.grouped_products_in_tensor_memory and T >= self.FUSED_TOKENS
                and self.one_group.numel() * tile >= T):
            ops.gemm_tn_tcgen05_grouped(x, self.up.weight.view(1, I, H), h, self.one_group, act=self.spec.activation,
                                        tile_rows=tile)
        else:
            z = self.up(ctx, x, "dense.z", out_dtype=torch.float32)
            ops.activation(z, h, self.spec.activation)
        return self.down(ctx, h, "dense.down")
