"""The gated delta rule with a decay per head and key channel: a recurrent mixer with a matrix of state
S [head_dim, v_head_dim] per head.

Per token and head, with q and k unit vectors (q also divided by sqrt(head_dim)), q, k and v behind a short causal
convolution over time and silu, beta = logistic(W_b x), g = exp(-exp(A_h) softplus(W_a2 W_a1 x + dt_bias)):

    S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

what a token writes is in its own read-out.  o is RMS-normed per head, scaled by a weight shared by the heads and by
logistic(W_g2 W_g1 x), then projected.  Value head h reads q / k head h // (heads / kv_heads).

One stacked projection gives q | k | v | beta | decay's and gate's low-rank parts, a second, block-diagonal one, gives
decay | gate from the latter.  What a request carries from token to token is a fixed-size float32 state in the
request's slot: S of every head and the last taps - 1 inputs of every convolved channel.  It starts at zero (the engine
zeroes a slot for its new occupant) and is put back when a step fails (the engine's snapshot).
"""
from __future__ import annotations

from typing import List

import torch

from ..cache.manager import FIXED_STATE
from ..config.spec import ChannelDeltaSpec, RunStep
from ..errors import WeightError
from ..kernels import ops
from ..weights.loader import MATRIX, VECTOR, TensorDecl
from .base import CacheNeed, Part, register_mixer
from .linear import Linear


def block_diagonal(a: torch.Tensor, b: torch.Tensor, multiple: int) -> torch.Tensor:
    """[[a, 0], [0, b]] with columns of zeros up to a multiple (tensor-core products want aligned rows)."""
    cols = a.shape[1] + b.shape[1]
    out = torch.zeros((a.shape[0] + b.shape[0], -(-cols // multiple) * multiple), dtype=a.dtype, device=a.device)
    out[:a.shape[0], :a.shape[1]] = a
    out[a.shape[0]:, a.shape[1]:cols] = b
    return out


@register_mixer("channel_delta")
class ChannelDelta(Part):
    def __init__(self, spec: ChannelDeltaSpec, prefix: str, tensors: dict, mctx):
        self.spec = s = spec
        p, nm = prefix, spec.names
        for down, up in ((nm.decay_down, nm.decay_up), (nm.gate_down, nm.gate_up)):
            if tensors[p + down].shape[0] != tensors[p + up].shape[1]:
                raise WeightError(f"tensors {p + down} and {p + up} disagree about their rank: "
                                  f"{tensors[p + down].shape[0]} and {tensors[p + up].shape[1]}")
        up = block_diagonal(tensors[p + nm.decay_up], tensors[p + nm.gate_up], 8)
        self.low_up = Linear(up, p + "a2_g2")
        stacked = [tensors[p + n] for n in (nm.q, nm.k, nm.v, nm.beta, nm.decay_down, nm.gate_down)]
        self.rank = up.shape[1]                    # of both low-rank parts together, in whole eights
        filler = self.rank - stacked[-2].shape[0] - stacked[-1].shape[0]
        if filler:
            stacked.append(torch.zeros((filler, s.hidden_size), dtype=stacked[0].dtype, device=stacked[0].device))
        self.proj = Linear(torch.cat(stacked, dim=0).contiguous(), p + "q_k_v_b_a1_g1")
        self.channels = 2 * s.kv_heads * s.head_dim + s.heads * s.v_head_dim
        self.conv_w = torch.cat([tensors[p + n + nm.conv_suffix] for n in (nm.q, nm.k, nm.v)], dim=0).float().contiguous()
        self.decay_log, self.decay_bias = tensors[p + nm.decay_log], tensors[p + nm.decay_bias]
        self.out_norm_w = tensors[p + nm.out_norm]
        self.out = Linear(tensors[p + nm.o], p + nm.o)

    @classmethod
    def tensor_decls(cls, s: ChannelDeltaSpec, prefix: str) -> List[TensorDecl]:
        p, nm = prefix, s.names
        qk, v = s.kv_heads * s.head_dim, s.heads * s.v_head_dim
        decls = []
        for n, rows in ((nm.q, qk), (nm.k, qk), (nm.v, v)):
            decls += [TensorDecl(p + n, (rows, s.hidden_size), MATRIX),
                      TensorDecl(p + n + nm.conv_suffix, (rows, s.conv_taps), VECTOR)]
        return decls + [TensorDecl(p + nm.beta, (s.heads, s.hidden_size), MATRIX),
                        TensorDecl(p + nm.decay_down, (None, s.hidden_size), MATRIX),
                        TensorDecl(p + nm.decay_up, (s.heads * s.head_dim, None), MATRIX),
                        TensorDecl(p + nm.decay_log, (s.heads,), VECTOR),
                        TensorDecl(p + nm.decay_bias, (s.heads * s.head_dim,), VECTOR),
                        TensorDecl(p + nm.gate_down, (None, s.hidden_size), MATRIX),
                        TensorDecl(p + nm.gate_up, (v, None), MATRIX),
                        TensorDecl(p + nm.out_norm, (s.v_head_dim,), VECTOR),
                        TensorDecl(p + nm.o, (s.hidden_size, v), MATRIX)]

    @staticmethod
    def state_size(s: ChannelDeltaSpec) -> int:
        channels = 2 * s.kv_heads * s.head_dim + s.heads * s.v_head_dim
        size = s.heads * s.head_dim * s.v_head_dim + channels * (s.conv_taps - 1)
        return -(-size // 4) * 4                   # every slot's row starts on 16 bytes

    @classmethod
    def cache_need_of(cls, s: ChannelDeltaSpec) -> CacheNeed:
        return CacheNeed(FIXED_STATE, state_shape=(cls.state_size(s),), state_dtype=torch.float32)

    def forward(self, ctx, x: torch.Tensor, run_step: RunStep, out_dtype=None) -> torch.Tensor:
        """-> [T, hidden] in ``out_dtype`` (default: the activation dtype)."""
        s = self.spec
        T = x.shape[0]
        proj = self.proj(ctx, x, "channel_delta.proj", out_dtype=torch.float32)
        rank = ctx.workspace.get("channel_delta.low_in", T, self.rank, ctx.dtype)
        ops.cast_columns(proj, self.channels + s.heads, rank)
        low = self.low_up(ctx, rank, "channel_delta.low", out_dtype=torch.float32)      # decay | gate
        state = ctx.cache.state_of_entry(run_step.cache)                                # [slots, state_size]
        gated = ctx.workspace.get("channel_delta.gated", T, s.heads * s.v_head_dim, ctx.dtype)
        ops.channel_delta(ctx, proj, self.conv_w, low, self.decay_log, self.decay_bias, state, self.out_norm_w, s.norm_eps,
                          gated, s.heads, s.kv_heads, s.head_dim, s.v_head_dim, s.conv_taps, s.unit_eps)
        return self.out(ctx, gated, "channel_delta.out", out_dtype=out_dtype)
