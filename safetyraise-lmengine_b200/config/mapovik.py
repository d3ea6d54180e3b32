"""Mapovik: config.json keys -> ModelSpec.

A Mapovik model is a list of pre-norm layers (layer norm without a bias) whose sublayers join the stream times
``residual_mult``.  ``loop`` {start, stop, times} repeats layers start .. stop - 1 with the same weights, every pass on
cache entries of its own; each pass begins with a product of the stream beside the embedded tokens (``loop.in``) and
the addition of the pass's own vector (``loop.step``).  ``type`` names a layer's mixer:

* ``parallel``: two mixers side by side on the same input -- ``left``, rotated attention (pairs (i, i + dims/2) of the
  first ``rot.dims`` elements, frequencies divided by ``rot.scaling.factor``); ``right``, a state space with one decay a
  head -- each output RMS-normed with a plain weight, then averaged.
* ``channel_delta``: the gated delta rule with a decay per head and key channel; the ranks of its two low-rank
  projections are the tensors'.

``mlp`` is null, ``kind: dense`` (no gate, squared activation) or ``kind: moe``: gated experts named by a table of token
ids.  The output head has a table of its own and its logits are multiplied by ``logit_scale``.  Tensor names: ``embed``,
``loop.in``, ``loop.step``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.mlp.*``, ``final.norm``, ``head``.  No
key has a default: what config.json does not give, the model does not have.
"""
from __future__ import annotations

import math

from ..errors import ConfigError, Unsupported
from .spec import (ChannelDeltaSpec, DenseSpec, LayerSpec, ModelSpec, NormSpec, PositionSpec, RotatedAttentionNames,
                   RotatedAttentionSpec, RoutedExpertsSpec, RunStep, SideBySideSpec, StateSpaceNames, StateSpaceSpec)

ARCHITECTURE = "Mapovik"
MAX_LAYERS = 4096
MAX_RUNS = 1 << 16
MAX_POSITIONS = 1 << 24       # the design sets no limit; angles are formed in double precision
UNIT_EPS = 1e-6               # fixed by the design: inside the root that makes q and k unit vectors


def _int(d: dict, key: str, where: str, least: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"config.json: {where}{key!r} must be an integer of at least {least}, got {v!r}")
    return v


def _real(d: dict, key: str, where: str) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v):
        raise ConfigError(f"config.json: {where}{key!r} must be a finite number, got {v!r}")
    return float(v)


def _num(d: dict, key: str, where: str) -> float:
    v = _real(d, key, where)
    if v <= 0:
        raise ConfigError(f"config.json: {where}{key!r} must be a finite positive number, got {v!r}")
    return v


def _obj(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}{key!r} must be an object")
    return v


def _shared(many: int, few: int, what: str, where: str) -> None:
    if many % few:
        raise ConfigError(f"config.json: {where}heads {many} is not a multiple of {what} {few}")


def _position(m: dict, dim: int, where: str):
    if m.get("rot") is None:
        return None
    rot, w = _obj(m, "rot", where), where + "rot."
    dims = _int(rot, "dims", w)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {w}dims {dims} must be even and at most the head size {dim}")
    divisor = 1.0
    if rot.get("scaling") is not None:
        scaling = _obj(rot, "scaling", w)
        if set(scaling) != {"factor"}:
            raise Unsupported(f"config.json: {w}scaling has the keys {sorted(scaling)}; a Mapovik rotation is scaled by one "
                              f"'factor'")
        divisor = _num(scaling, "factor", w + "scaling.")
    return PositionSpec("rotary_half", theta=_num(rot, "base", w), rotary_dim=dims, head_dim=dim, divisor=divisor)


def _attention(m: dict, width: int, where: str, p: str) -> RotatedAttentionSpec:
    heads, kv, dim = _int(m, "heads", where), _int(m, "kv_heads", where), _int(m, "dim", where)
    _shared(heads, kv, "kv_heads", where)
    return RotatedAttentionSpec(
        kind="rotated_attention", hidden_size=width, heads=heads, kv_heads=kv, head_dim=dim, v_head_dim=_int(m, "vdim", where),
        softmax_scale=_num(m, "scale", where), position=_position(m, dim, where),
        names=RotatedAttentionNames(p + "q", p + "k", p + "v", p + "o", ".b"))


def _state_space(m: dict, width: int, eps: float, where: str, p: str) -> StateSpaceSpec:
    heads, groups, vdim = _int(m, "heads", where), _int(m, "groups", where), _int(m, "vdim", where)
    _shared(heads, groups, "groups", where)
    parts = _int(m, "norm_groups", where)
    if heads * vdim % parts:
        raise ConfigError(f"config.json: {where}heads * vdim = {heads * vdim} is not a multiple of norm_groups {parts}")
    return StateSpaceSpec(
        kind="state_space", hidden_size=width, heads=heads, head_dim=vdim, state=_int(m, "state", where), groups=groups,
        norm_parts=parts, conv_taps=_int(m, "conv", where), norm_eps=eps,
        names=StateSpaceNames(p + "in", p + "conv", p + "dt_bias", p + "A_log", p + "D", p + "norm", p + "o"))


def _channel_delta(m: dict, width: int, eps: float, where: str) -> ChannelDeltaSpec:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    _shared(heads, kv, "kv_heads", where)
    return ChannelDeltaSpec(kind="channel_delta", hidden_size=width, heads=heads, kv_heads=kv, head_dim=_int(m, "dim", where),
                            v_head_dim=_int(m, "vdim", where), conv_taps=_int(m, "conv", where), norm_eps=eps,
                            unit_eps=UNIT_EPS)


def _feed_forward(mlp: dict, width: int, vocab: int, where: str):
    kind = mlp.get("kind")
    if kind == "dense":
        return DenseSpec("dense", width, _int(mlp, "ff", where), "relu_squared")
    if kind != "moe":
        raise Unsupported(f"config.json: {where}kind {kind!r}: a Mapovik feed-forward is 'dense' or 'moe'")
    router = _obj(mlp, "router", where)
    experts, top = _int(router, "experts", where + "router."), _int(router, "top", where + "router.")
    if top > experts:
        raise ConfigError(f"config.json: {where}router.top {top} exceeds router.experts {experts}")
    return RoutedExpertsSpec("routed_experts", width, _int(_obj(mlp, "expert", where), "ff", where + "expert."), "silu",
                             experts=experts, top=top, router_bias=False, scoring="table", vocab=vocab)


def read_spec(root: dict) -> ModelSpec:
    if root.get("architecture") != ARCHITECTURE:
        raise ConfigError(f"config.json: architecture {root.get('architecture')!r} is not {ARCHITECTURE}")
    width, vocab = _int(root, "width", ""), _int(root, "vocab", "")
    eps = _num(_obj(root, "norm", ""), "eps", "norm.")
    mult, logit_scale = _real(root, "residual_mult", ""), _real(root, "logit_scale", "")
    entries = root.get("layers")
    if not isinstance(entries, list) or not entries or len(entries) > MAX_LAYERS:
        raise ConfigError(f"config.json: 'layers' must list 1 to {MAX_LAYERS} layers")
    norm = NormSpec("layernorm", width, eps)
    layers = []
    for i, entry in enumerate(entries):
        where = f"layers[{i}]."
        if not isinstance(entry, dict) or not isinstance(entry.get("type"), str):
            raise ConfigError(f"config.json: {where[:-1]} must be an object with a 'type'")
        m, w = _obj(entry, "mixer", where), where + "mixer."
        if entry["type"] == "parallel":
            left = _attention(_obj(m, "left", w), width, w + "left.", "mix.left.")
            right = _state_space(_obj(m, "right", w), width, eps, w + "right.", "mix.right.")
            mixer = SideBySideSpec(kind="side_by_side", hidden_size=width, mixers=(left, right),
                                   out_norm_names=("mix.left.out", "mix.right.out"), out_norm_eps=eps)
        elif entry["type"] == "channel_delta":
            mixer = _channel_delta(m, width, eps, w)
        else:
            raise Unsupported(f"config.json: {where[:-1]} has type {entry['type']!r}; a Mapovik layer is 'parallel' or "
                              f"'channel_delta'")
        ff = _feed_forward(_obj(entry, "mlp", where), width, vocab, where + "mlp.") if entry.get("mlp") is not None else None
        layers.append(LayerSpec(block="pre_norm", mixer=mixer, feed_forward=ff, mixer_norm=norm,
                                feed_forward_norm=norm if ff else None, weight_prefix=f"l{i}.", mixer_norm_name="norm1",
                                feed_forward_norm_name="norm2", sublayer_scale=mult))

    runs = [(i, None) for i in range(len(layers))]
    if root.get("loop") is not None:
        loop = _obj(root, "loop", "")
        start, stop = _int(loop, "start", "loop.", least=0), _int(loop, "stop", "loop.")
        times = _int(loop, "times", "loop.")
        if not start < stop <= len(layers):
            raise ConfigError(f"config.json: loop {start} .. {stop} does not lie within the {len(layers)} layers")
        if (stop - start) * times > MAX_RUNS:
            raise ConfigError(f"config.json: {times} passes over {stop - start} layers exceed {MAX_RUNS} layer runs")
        runs[start:stop] = [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
    run_order, entry = [], 0
    for i, begins in runs:                     # each run of a layer has cache entries of its own: one for each of its mixers
        n = len(layers[i].mixer.mixers) if isinstance(layers[i].mixer, SideBySideSpec) else 1
        run_order.append(RunStep(i, entry, True, more_caches=tuple(range(entry + 1, entry + n)), begins_pass=begins))
        entry += n
    return ModelSpec(architecture=ARCHITECTURE, hidden_size=width, vocab_size=vocab,
                     max_position_embeddings=MAX_POSITIONS, layers=tuple(layers), run_order=tuple(run_order),
                     final_norm=norm, tie_word_embeddings=False, eos_token_ids=(), embed_name="embed",
                     final_norm_name="final.norm", head_name="head", logit_scale=logit_scale)
