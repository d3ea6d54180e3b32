"""The decoder: embedding, blocks in their run order, final norm, output head.

Built from a ``ModelSpec`` alone; which architecture the spec came from does
not matter here.  src/model/native.rs:156-312.
"""
from __future__ import annotations

from collections import OrderedDict
from typing import Dict, List

import torch

from ..cache.manager import FIXED_STATE, CacheGroupSpec
from ..config.spec import ModelSpec
from ..errors import ConfigError
from ..kernels import ops
from ..weights.loader import MATRIX, TABLE, VECTOR, TensorDecl, load_tensors
from .base import (BLOCKS, EMBEDDING, FAULT_ACTIVATION, FAULT_TOKEN, NORMS, POSITION_ENCODINGS, STATUS_WORDS,
                   ModelContext, lookup, split_delta)
from .linear import Linear


def tensor_decls(spec: ModelSpec) -> List[TensorDecl]:
    decls = [TensorDecl(spec.embed_name, (spec.vocab_size, spec.hidden_size), TABLE)]
    if spec.embed_position is not None:
        decls += lookup(POSITION_ENCODINGS, spec.embed_position.kind, "position encoding").tensor_decls(
            spec.embed_position, spec.embed_position_name)
    if spec.embed_norm is not None:
        decls += lookup(NORMS, spec.embed_norm.kind, "norm").tensor_decls(spec.embed_norm, spec.embed_norm_name)
    for layer in spec.layers:
        decls += lookup(BLOCKS, layer.block, "block").tensor_decls(layer)
    decls += lookup(NORMS, spec.final_norm.kind, "norm").tensor_decls(spec.final_norm, spec.final_norm_name)
    if spec.num_passes:
        H = spec.hidden_size
        decls += [TensorDecl(spec.pass_product_name, (H, 2 * H), MATRIX),
                  TensorDecl(spec.pass_vectors_name, (spec.num_passes, H), VECTOR)]
    if not spec.tie_word_embeddings:
        decls.append(TensorDecl(spec.head_name, (spec.vocab_size, spec.hidden_size), MATRIX))
    return decls


def cache_groups_of(spec: ModelSpec) -> List[CacheGroupSpec]:
    """What a model of this specification needs from the cache manager, from the specification alone.
    Run steps with equal needs share a group; each group gets pages (or state) of its own."""
    from .base import MIXERS

    def needs_of(step):
        """(need, cache entry) of every mixer of the step: one, or one per mixer of a side-by-side pair."""
        mixer = spec.layers[step.layer].mixer
        need = lookup(MIXERS, mixer.kind, "mixer").cache_need_of(mixer)
        needs = need if isinstance(need, tuple) else (need,)
        entries = (step.cache,) + tuple(step.more_caches)
        if len(needs) != len(entries):
            raise ConfigError(f"a run step of layer {step.layer} names {len(entries)} cache entries for {len(needs)} mixers")
        return list(zip(needs, entries))

    by_need: "OrderedDict[object, list]" = OrderedDict()
    owner_need = {}
    for step in spec.run_order:
        for need, entry in needs_of(step):
            if need.kind == "none":
                continue
            if step.writes_cache:
                if entry in owner_need:
                    raise ConfigError(f"cache entry {entry} is written by two run steps")
                owner_need[entry] = need
                by_need.setdefault(need, []).append(entry)
    for step in spec.run_order:
        for need, entry in needs_of(step):
            if need.kind != "none" and not step.writes_cache and owner_need.get(entry) != need:
                raise ConfigError(f"a run step reads cache entry {entry}, which no step with the "
                                  f"same needs writes")
    groups = []
    for i, (need, entries) in enumerate(by_need.items()):
        groups.append(CacheGroupSpec(name=f"g{i}:{need.kind}", kind=need.kind, entries=tuple(entries),
                                     kv_heads=need.kv_heads, head_dim=need.head_dim, window=need.window,
                                     state_shape=need.state_shape, state_dtype=need.state_dtype,
                                     v_head_dim=need.v_head_dim, keep_first=need.keep_first))
    return groups


class DecoderModel:
    def __init__(self, spec: ModelSpec, mctx: ModelContext, source):
        self.spec, self.mctx = spec, mctx
        tensors = load_tensors(source, tensor_decls(spec), mctx.dtype, mctx.device)
        self.embed = tensors[spec.embed_name]
        self.embed_position = None
        if spec.embed_position is not None:
            cls = lookup(POSITION_ENCODINGS, spec.embed_position.kind, "position encoding")
            if getattr(cls, "applies", None) != EMBEDDING:
                raise ConfigError(f"position encoding {spec.embed_position.kind!r} does not add to the embedding")
            self.embed_position = cls(spec.embed_position, mctx, tensors, spec.embed_position_name)
        self.embed_norm = None
        if spec.embed_norm is not None:
            self.embed_norm = lookup(NORMS, spec.embed_norm.kind, "norm")(spec.embed_norm, spec.embed_norm_name,
                                                                          tensors, mctx)
        self.blocks = [lookup(BLOCKS, layer.block, "block")(layer, tensors, mctx) for layer in spec.layers]
        self.final_norm = lookup(NORMS, spec.final_norm.kind, "norm")(spec.final_norm, spec.final_norm_name,
                                                                      tensors, mctx)
        # tied: the head IS the embedding table (same storage), src/model/native.rs:171-179
        self.head = Linear(self.embed if spec.tie_word_embeddings else tensors[spec.head_name], "lm_head")
        if spec.logit_scale != 1.0:      # on the final norm's weight: head (c n) = c (head n), and the weight is float32
            if spec.final_norm.unit_offset:
                raise ConfigError("a factor on the logits needs a final norm whose weight is applied as it is")
            self.final_norm.weight = self.final_norm.weight * spec.logit_scale
        self.pass_product = self.pass_vectors = None
        if spec.num_passes:
            w, H = tensors[spec.pass_product_name], spec.hidden_size
            if mctx.dtype == torch.bfloat16:       # the stream's two halves meet the same columns
                w = torch.cat([w[:, :H], w], dim=1)
            self.pass_product = Linear(w.contiguous(), spec.pass_product_name)
            self.pass_vectors = tensors[spec.pass_vectors_name]
        self.keeps_embedding = any(s.add_embedding or s.begins_pass is not None for s in spec.run_order) and \
            (self.embed_norm is not None or self.embed_position is not None)
        for step in spec.run_order:
            if not 0 <= step.layer < len(self.blocks):
                raise ConfigError(f"run order names layer {step.layer}, the model has {len(self.blocks)}")
        self.status = torch.zeros(STATUS_WORDS, dtype=torch.int32, device=mctx.device)   # when a step brings none
        # decode steps may be replayed from CUDA graphs only if no part plans on the host
        self.replayable = all(getattr(b, "replayable", True) for b in self.blocks) and \
            getattr(self.final_norm, "replayable", True) and getattr(self.embed_position, "replayable", True)

    def cache_groups(self) -> List[CacheGroupSpec]:
        return cache_groups_of(self.spec)

    def forward(self, ctx) -> torch.Tensor:
        """Runs the tokens of ``ctx``; returns float32 logits [len(ctx.logit_rows), vocab]."""
        H = self.spec.hidden_size
        residual = ctx.workspace.get("residual", ctx.T, H, torch.float32)
        status = ctx.status if ctx.status is not None else self.status
        if self.embed_norm is not None:
            # the stream starts from the normed rows of the table: gathered beside it, normed into it (float32)
            rows = ctx.workspace.get("embed.rows", ctx.T, H, torch.float32)
            ops.embed_gather(ctx.token_ids, self.embed, rows, status[FAULT_TOKEN:FAULT_TOKEN + 1], scale=self.spec.embed_scale)
            self.embed_norm.apply(rows, None, residual)
        else:
            ops.embed_gather(ctx.token_ids, self.embed, residual, status[FAULT_TOKEN:FAULT_TOKEN + 1], scale=self.spec.embed_scale)
        if self.embed_position is not None:
            self.embed_position.add_to_embedding(ctx, residual)
        kept = None
        if self.keeps_embedding:         # more than the table's rows: a later step needs a copy of what the embedding left
            kept = ctx.workspace.get("embed.kept", ctx.T, H, torch.float32)
            ops.cast(residual, kept)
        pending = None
        order = self.spec.run_order
        for i, step in enumerate(order):
            if step.begins_pass is not None:
                pending = self._begin_pass(ctx, residual, pending, kept, step.begins_pass)
            if step.add_embedding:
                if kept is not None:
                    ops.residual_add(residual, kept)
                else:                    # the rows themselves, read from the table again
                    ops.embed_gather(ctx.token_ids, self.embed, residual, status[FAULT_TOKEN:FAULT_TOKEN + 1],
                                     scale=self.spec.embed_scale, add=True)
            # a block ahead of an addition to the stream prepares no input: what it leaves is pending or in the stream
            nxt = order[i + 1] if i + 1 < len(order) else None
            nxt = self.blocks[nxt.layer] if nxt is not None and not nxt.add_embedding and nxt.begins_pass is None else None
            pending = self.blocks[step.layer].forward(ctx, residual, pending, step, nxt)
        # NaN and infinity stay in a residual stream that is only ever added to, and every key or value
        # a step writes is read by its own token: one look at the end covers every block
        # (src/model/native.rs:276-278, src/engine/state.rs:56-58)
        left, _ = split_delta(pending)
        ops.check_finite(residual, left if isinstance(left, torch.Tensor) else None,
                         status[FAULT_ACTIVATION:FAULT_ACTIVATION + 1])
        R = ctx.logit_rows.shape[0]
        logits = ctx.workspace.get("logits", R, self.spec.vocab_size, torch.float32, reserve=64)
        if R == 0:          # nothing wanted: the step only had to fill the cache
            return logits
        hn = ctx.workspace.get("final.normed", R, H, ctx.dtype, reserve=64)
        self.final_norm.apply(residual, pending, hn, rows=ctx.logit_rows)
        self.head.into(ctx, hn, logits)
        if self.spec.logit_softcap is not None:
            ops.softcap(logits, self.spec.logit_softcap)
        return logits

    def _begin_pass(self, ctx, residual, pending, kept, index: int):
        """x <- W [x; x_0] + v_index, in place; what was pending is part of x.  -> None: nothing is pending behind it."""
        T, H = residual.shape
        delta, scale = split_delta(pending)
        low = ctx.dtype == torch.bfloat16
        both = ctx.workspace.get("pass.both", T, (3 if low else 2) * H, ctx.dtype)
        ops.stream_beside_embedding(residual, delta, scale, ctx.token_ids, self.embed, self.spec.embed_scale, kept, both)
        self.pass_product.into(ctx, both, residual)
        ops.add_row(residual, self.pass_vectors[index])
        return None

    def weight_bytes(self) -> int:
        seen, total = set(), 0
        def walk(obj):
            nonlocal total
            if isinstance(obj, torch.Tensor):
                key = obj.untyped_storage().data_ptr()
                if key not in seen:
                    seen.add(key)
                    total += obj.numel() * obj.element_size()
            elif isinstance(obj, (list, tuple)):
                for o in obj:
                    walk(o)
            elif hasattr(obj, "__dict__"):
                for k, o in vars(obj).items():
                    if k not in ("mctx", "spec", "options"):
                        walk(o)
        walk(self)
        return total
