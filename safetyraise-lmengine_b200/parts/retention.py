"""Retention: a linear attention with a matrix of state S [head_dim, v_head_dim] per head that fades at a fixed rate.

    q = R(W_q h);  k = R(W_k h) / sqrt(head_dim);  v = W_v h        R: the rotary encoding on a head's leading elements
    S <- decay_h S + k v^T;   o = S^T q
    out = W_o (U(o) * silu(W_g h))                                  U: each head over its root mean square, no weight

One stacked projection gives q | k | v | gate in float32; rotation, state, read-out and norm are float32.  The state is a
fixed-size float32 row of the request's slot: zero for a new request, carried from token to token, put back when a step
fails.
"""
from __future__ import annotations

from typing import List

import torch

from ..cache.manager import FIXED_STATE
from ..config.spec import RetentionSpec, RunStep
from ..errors import ConfigError
from ..kernels import ops
from ..weights.loader import MATRIX, TensorDecl
from .base import POSITION_ENCODINGS, ROTATION, CacheNeed, Part, lookup, register_mixer
from .linear import Linear


@register_mixer("retention")
class Retention(Part):
    def __init__(self, spec: RetentionSpec, prefix: str, tensors: dict, mctx):
        self.spec = s = spec
        p, nm = prefix, spec.names
        if len(s.decay) != s.heads:
            raise ConfigError(f"retention: {len(s.decay)} decays for {s.heads} heads")
        self.proj = Linear(torch.cat([tensors[p + n] for n in (nm.q, nm.k, nm.v, nm.gate)], dim=0).contiguous(), p + "q_k_v_g")
        self.decay = torch.tensor(s.decay, dtype=torch.float32, device=mctx.device)
        self.position = None
        if s.position is not None:
            cls = lookup(POSITION_ENCODINGS, s.position.kind, "position encoding")
            if getattr(cls, "applies", None) != ROTATION:
                raise ConfigError(f"position encoding {s.position.kind!r} is not a rotation")
            self.position = cls(s.position, mctx)
        self.out = Linear(tensors[p + nm.o], p + nm.o)

    @classmethod
    def tensor_decls(cls, s: RetentionSpec, prefix: str) -> List[TensorDecl]:
        p, nm = prefix, s.names
        qk, v = s.heads * s.head_dim, s.heads * s.v_head_dim
        return [TensorDecl(p + nm.q, (qk, s.hidden_size), MATRIX), TensorDecl(p + nm.k, (qk, s.hidden_size), MATRIX),
                TensorDecl(p + nm.v, (v, s.hidden_size), MATRIX), TensorDecl(p + nm.gate, (v, s.hidden_size), MATRIX),
                TensorDecl(p + nm.o, (s.hidden_size, v), MATRIX)]

    @classmethod
    def cache_need_of(cls, s: RetentionSpec) -> CacheNeed:
        return CacheNeed(FIXED_STATE, state_shape=(s.heads * s.head_dim * s.v_head_dim,), state_dtype=torch.float32)

    def forward(self, ctx, x: torch.Tensor, run_step: RunStep) -> torch.Tensor:
        s = self.spec
        proj = self.proj(ctx, x, "retention.proj", out_dtype=torch.float32)
        rotation = self.position.rotation(ctx) if self.position is not None else None
        gated = ctx.workspace.get("retention.out", x.shape[0], s.heads * s.v_head_dim, ctx.dtype)
        ops.retention(ctx, proj, rotation, self.decay, s.norm_eps, ctx.cache.state_of_entry(run_step.cache), gated, s.heads,
                      s.head_dim, s.v_head_dim)
        return self.out(ctx, gated, "retention.proj_out")
