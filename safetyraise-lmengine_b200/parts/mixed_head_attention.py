"""Grouped-query attention whose heads exchange their weights behind the softmax, with a learned bias by distance and a
sliding window that keeps the sequence's first tokens:

    q, k, v = W h;   q, k <- N(w, .) over all their heads at once                        (when the spec gives an eps)
    s_h(i, j) = (q_i . k_j) * scale + bias[bucket(i - j), h],   0 <= i - j and (i - j < window or j < keep_first)
    p_h = softmax_j(s_h);   w_h = sum_g mix[h, g] p_g;   out_h = (sum_j w_h v_j) * logistic(W_g h)     (gate per element)

The buckets' table is spread over distances once, when the part is built: a score looks its bias up by min(i - j, max).
One stacked projection gives q | k | v | gate logits in float32, so norms, scores and gates see unrounded values; keys
and values go to the pages in the cache's dtype.
"""
from __future__ import annotations

from fractions import Fraction
from typing import List

import torch

from ..cache.manager import PAGED_ALL, PAGED_WINDOW
from ..config.spec import MixedHeadAttentionSpec, RunStep
from ..errors import ConfigError, WeightError
from ..kernels import ops
from ..weights.loader import MATRIX, VECTOR, TensorDecl
from .base import CacheNeed, Part, register_mixer
from .linear import Linear


def distance_buckets(rows: int, farthest: float) -> List[int]:
    """The bucket of every distance 0 .. ceil(farthest) (farther ones share the last): with h = rows / 2, n < h has a
    bucket of its own, n >= h falls into min(rows - 1, h + floor(ln(n / h) / ln(farthest / h) * (rows - h))).  The floor
    is taken exactly: bucket h + k begins where n^(rows - h) h^k >= farthest^k h^(rows - h)."""
    h = rows // 2
    if rows < 2 or rows % 2:
        raise WeightError(f"a bias by distance needs an even number of rows, got {rows}")
    D = Fraction(farthest)
    if D <= h:
        raise ConfigError(f"the farthest bucketed distance {farthest} must exceed half of the {rows} bias rows")
    last = -(-D.numerator // D.denominator)
    out, k = [], 0
    ratio = D / h
    starts = [ratio ** i * Fraction(h) ** (rows - h) for i in range(rows - h)]      # bucket h + i: n^(rows - h) from here on
    for n in range(last + 1):
        if n < h:
            out.append(n)
            continue
        power = Fraction(n) ** (rows - h)
        while k + 1 < rows - h and power >= starts[k + 1]:
            k += 1
        out.append(h + k)
    return out


@register_mixer("mixed_head_attention")
class MixedHeadAttention(Part):
    def __init__(self, spec: MixedHeadAttentionSpec, prefix: str, tensors: dict, mctx):
        self.spec = spec
        p, nm = prefix, spec.names
        rows = [tensors[p + nm.q], tensors[p + nm.k], tensors[p + nm.v]]
        if spec.output_gate:
            rows.append(tensors[p + nm.gate])
        self.proj = Linear(torch.cat(rows, dim=0).contiguous(), p + "qkvg")
        self.gate_offset = spec.heads * spec.head_dim + spec.kv_heads * (spec.head_dim + spec.v_head_dim)
        self.q_norm = self.k_norm = None
        if spec.qk_norm_eps is not None:
            self.q_norm, self.k_norm = tensors[p + nm.q_norm], tensors[p + nm.k_norm]
        self.bias = None                                     # float32 [heads, distances]
        if spec.bias_max is not None:
            table = tensors[p + nm.distance_bias].float()
            ids = torch.tensor(distance_buckets(table.shape[0], spec.bias_max), device=table.device)
            self.bias = table[ids].t().contiguous()
        self.mix = tensors[p + nm.head_mix].float().contiguous() if spec.head_mix else None
        self.mix_low = self.mix is not None and not bool((self.mix.bfloat16().float() == self.mix).all())
        self.out = Linear(tensors[p + nm.o], p + nm.o)

    @classmethod
    def tensor_decls(cls, s: MixedHeadAttentionSpec, prefix: str) -> List[TensorDecl]:
        p, nm = prefix, s.names
        qd, kd, od = s.heads * s.head_dim, s.kv_heads * s.head_dim, s.heads * s.v_head_dim
        decls = [TensorDecl(p + nm.q, (qd, s.hidden_size), MATRIX), TensorDecl(p + nm.k, (kd, s.hidden_size), MATRIX),
                 TensorDecl(p + nm.v, (s.kv_heads * s.v_head_dim, s.hidden_size), MATRIX)]
        if s.qk_norm_eps is not None:
            decls += [TensorDecl(p + nm.q_norm, (qd,), VECTOR), TensorDecl(p + nm.k_norm, (kd,), VECTOR)]
        if s.bias_max is not None:
            decls.append(TensorDecl(p + nm.distance_bias, (None, s.heads), MATRIX))
        if s.head_mix:
            decls.append(TensorDecl(p + nm.head_mix, (s.heads, s.heads), MATRIX))
        if s.output_gate:
            decls.append(TensorDecl(p + nm.gate, (od, s.hidden_size), MATRIX))
        decls.append(TensorDecl(p + nm.o, (s.hidden_size, od), MATRIX))
        return decls

    @classmethod
    def cache_need_of(cls, s: MixedHeadAttentionSpec) -> CacheNeed:
        return CacheNeed(PAGED_WINDOW if s.window else PAGED_ALL, s.kv_heads, s.head_dim, s.window,
                         v_head_dim=None if s.v_head_dim == s.head_dim else s.v_head_dim,
                         keep_first=s.keep_first if s.window else 0)

    def forward(self, ctx, x: torch.Tensor, run_step: RunStep) -> torch.Tensor:
        s = self.spec
        T = x.shape[0]
        proj = self.proj(ctx, x, "mixed_attn.proj", out_dtype=torch.float32)
        k_pool, v_pool, group = ctx.cache.kv_of_entry(run_step.cache)
        q = ctx.workspace.get("mixed_attn.q", T, s.heads * s.head_dim,
                              ops.mixed_head_query_dtype(ctx.dtype, s.heads, s.kv_heads, s.head_dim, s.v_head_dim))
        ops.attention_wide_norm_append(proj, self.q_norm, self.k_norm, s.qk_norm_eps, q, k_pool, v_pool, ctx.kv_slot[group],
                                       s.heads, s.kv_heads, s.head_dim, s.v_head_dim, run_step.writes_cache)
        attended = ctx.workspace.get("mixed_attn.out", T, s.heads * s.v_head_dim, ctx.dtype)
        ops.mixed_head_attention(ctx, q, k_pool, v_pool, attended, ctx.block_tables[group], s.heads, s.kv_heads, s.head_dim,
                                 s.v_head_dim, s.softmax_scale, s.window or 0, s.keep_first, bias=self.bias, mix=self.mix,
                                 gate=(proj, self.gate_offset) if s.output_gate else None, mix_low=self.mix_low)
        return self.out(ctx, attended, "mixed_attn.o")
