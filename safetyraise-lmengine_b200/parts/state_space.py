"""A state space with one decay a head: a recurrent mixer with a matrix of state S [state, head_dim] per head.

    [z | x | B | C | dt] = W_in h;   x, B, C <- silu(conv(x, B, C) + b)     a short causal convolution per channel over time
    dt <- softplus(dt + dt_bias)                                            one step size a head
    S <- exp(-exp(A_h) dt) S + dt B x^T;   y = S^T C + D_h x                head h: B and C of group h // (heads / groups)
    out = W_o N(w, y * silu(z))                                             N: each of ``norm_parts`` equal parts by itself

The projection writes float32, so everything that enters the recurrence does so unrounded; the recurrence itself is
float32.  What a request carries from token to token is a fixed-size float32 state in the request's slot: S of every
head and the last taps - 1 inputs of every convolved channel.  It starts at zero (the engine zeroes a slot for its new
occupant) and is put back when a step fails (the engine's snapshot).
"""
from __future__ import annotations

from typing import List

import torch

from ..cache.manager import FIXED_STATE
from ..config.spec import RunStep, StateSpaceSpec
from ..kernels import ops
from ..weights.loader import MATRIX, VECTOR, TensorDecl
from .base import CacheNeed, Part, register_mixer
from .linear import Linear


@register_mixer("state_space")
class StateSpace(Part):
    def __init__(self, spec: StateSpaceSpec, prefix: str, tensors: dict, mctx):
        self.spec = spec
        p, nm = prefix, spec.names
        self.inp = Linear(tensors[p + nm.inp], p + nm.inp)
        self.conv_w, self.conv_b = tensors[p + nm.conv], tensors[p + nm.conv + ".b"]
        self.dt_bias, self.a_log, self.D = tensors[p + nm.dt_bias], tensors[p + nm.a_log], tensors[p + nm.d]
        self.out_norm_w = tensors[p + nm.out_norm]
        self.out = Linear(tensors[p + nm.o], p + nm.o)

    @staticmethod
    def _channels(s: StateSpaceSpec) -> int:
        return s.heads * s.head_dim + 2 * s.groups * s.state

    @classmethod
    def tensor_decls(cls, s: StateSpaceSpec, prefix: str) -> List[TensorDecl]:
        p, nm = prefix, s.names
        inner, channels = s.heads * s.head_dim, cls._channels(s)
        return [TensorDecl(p + nm.inp, (inner + channels + s.heads, s.hidden_size), MATRIX),
                TensorDecl(p + nm.conv, (channels, s.conv_taps), VECTOR),
                TensorDecl(p + nm.conv + ".b", (channels,), VECTOR),
                TensorDecl(p + nm.dt_bias, (s.heads,), VECTOR),
                TensorDecl(p + nm.a_log, (s.heads,), VECTOR),
                TensorDecl(p + nm.d, (s.heads,), VECTOR),
                TensorDecl(p + nm.out_norm, (inner,), VECTOR),
                TensorDecl(p + nm.o, (s.hidden_size, inner), MATRIX)]

    @classmethod
    def state_size(cls, s: StateSpaceSpec) -> int:
        size = s.heads * s.head_dim * s.state + cls._channels(s) * (s.conv_taps - 1)
        return -(-size // 4) * 4                   # every slot's row starts on 16 bytes

    @classmethod
    def cache_need_of(cls, s: StateSpaceSpec) -> CacheNeed:
        return CacheNeed(FIXED_STATE, state_shape=(cls.state_size(s),), state_dtype=torch.float32)

    def forward(self, ctx, x: torch.Tensor, run_step: RunStep, out_dtype=None) -> torch.Tensor:
        """-> [T, hidden] in ``out_dtype`` (default: the activation dtype)."""
        s = self.spec
        T, inner = x.shape[0], s.heads * s.head_dim
        proj = self.inp(ctx, x, "state_space.proj", out_dtype=torch.float32)
        state = ctx.cache.state_of_entry(run_step.cache)                    # [slots, state_size]
        y = ctx.workspace.get("state_space.y", T, inner, torch.float32)
        ops.state_space(ctx, proj, self.conv_w, self.conv_b, self.dt_bias, self.a_log, self.D, state, y, s.heads, s.groups,
                        s.state, s.head_dim, s.conv_taps)
        gated = ctx.workspace.get("state_space.gated", T, inner, ctx.dtype)
        ops.state_space_output(y, proj, self.out_norm_w, s.norm_eps, gated, s.norm_parts)
        return self.out(ctx, gated, "state_space.out", out_dtype=out_dtype)
