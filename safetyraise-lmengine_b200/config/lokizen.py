"""Lokizen: config.json keys -> ModelSpec.

A Lokizen model is a list of pre-norm layers, some of which may run several times in a row: ``loop`` {start, stop, times}
repeats layers start .. stop - 1 with the same weights, every pass on cache entries of its own; ahead of each pass but
the first the embedded tokens join the stream again.  ``type`` names a layer's mixer:

* ``attention``: grouped-query attention without a rotation, q and k normed over all heads at once, a learned bias per
  bucket of distances (``bias_max``; the number of buckets is the tensor's), a sliding window (``mask.size``) that keeps
  the sequence's first ``mask.keep_first`` tokens, heads that mix their weights behind the softmax, a gate per element.
* ``retention``: a linear attention whose state fades at a fixed rate per head (``decay``), with a rotation of the
  leading ``rot.dims`` elements of q and k.

``mlp`` is null or ``kind: moe``: ungated experts with a squared activation, chosen by logistic scores plus a learned
correction and weighted by the scores times ``router.scale``.  The embedded tokens are multiplied by
``embedding.scale``; the output head has a table of its own.  Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``,
``l<i>.norm2``, ``l<i>.mlp.*``, ``final.norm``, ``head``.  No key has a default: what config.json does not give, the
model does not have.
"""
from __future__ import annotations

import math

from ..errors import ConfigError, Unsupported
from .spec import (LayerSpec, MixedHeadAttentionSpec, ModelSpec, NormSpec, PositionSpec, RetentionSpec, RoutedExpertsSpec,
                   RunStep)

ARCHITECTURE = "Lokizen"
MAX_LAYERS = 4096
MAX_RUNS = 1 << 16
MAX_POSITIONS = 1 << 24       # the design sets no limit; angles are formed in double precision, distances are integers


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


def _attention(m: dict, width: int, eps: float, where: str) -> MixedHeadAttentionSpec:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads {heads} is not a multiple of kv_heads {kv}")
    window, keep = None, 0
    if m.get("mask") is not None:
        mask, w = _obj(m, "mask", where), where + "mask."
        window = _int(mask, "size", w)
        keep = _int(mask, "keep_first", w, least=0) if mask.get("keep_first") is not None else 0
    return MixedHeadAttentionSpec(
        kind="mixed_head_attention", hidden_size=width, heads=heads, kv_heads=kv, head_dim=_int(m, "dim", where),
        v_head_dim=_int(m, "vdim", where), softmax_scale=_num(m, "scale", where), qk_norm_eps=eps,
        bias_max=_num(m, "bias_max", where), window=window, keep_first=keep, head_mix=True, output_gate=True)


def _retention(m: dict, width: int, eps: float, where: str) -> RetentionSpec:
    heads, dim = _int(m, "heads", where), _int(m, "dim", where)
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != heads:
        raise ConfigError(f"config.json: {where}'decay' must list one number for each of the {heads} heads")
    decay = tuple(_real({"decay": v}, "decay", f"{where}decay[{h}] of ") for h, v in enumerate(decay))
    if any(not 0.0 <= v <= 1.0 for v in decay):
        raise ConfigError(f"config.json: {where}'decay' must lie between 0 and 1")
    position = None
    if m.get("rot") is not None:
        rot, w = _obj(m, "rot", where), where + "rot."
        dims = _int(rot, "dims", w)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {w}dims {dims} must be even and at most {dim}")
        position = PositionSpec("rotary_half", theta=_num(rot, "base", w), rotary_dim=dims, head_dim=dim)
    return RetentionSpec(kind="retention", hidden_size=width, heads=heads, head_dim=dim, v_head_dim=_int(m, "vdim", where),
                         decay=decay, position=position, norm_eps=eps)


def _feed_forward(mlp: dict, width: int, where: str) -> RoutedExpertsSpec:
    if mlp.get("kind") != "moe":
        raise Unsupported(f"config.json: {where}kind {mlp.get('kind')!r}: a Lokizen feed-forward is 'moe'")
    router = _obj(mlp, "router", where)
    experts, top = _int(router, "experts", where + "router."), _int(router, "top", where + "router.")
    if top > experts:
        raise ConfigError(f"config.json: {where}router.top {top} exceeds router.experts {experts}")
    return RoutedExpertsSpec("routed_experts", width, _int(_obj(mlp, "expert", where), "ff", where + "expert."),
                             "relu_squared", experts=experts, top=top, router_bias=False, scoring="logistic", gated=False,
                             correction=True, weight_scale=_real(router, "scale", where + "router."))


def read_spec(root: dict) -> ModelSpec:
    if root.get("architecture") != ARCHITECTURE:
        raise ConfigError(f"config.json: architecture {root.get('architecture')!r} is not {ARCHITECTURE}")
    width, vocab = _int(root, "width", ""), _int(root, "vocab", "")
    eps = _num(_obj(root, "norm", ""), "eps", "norm.")
    scale = _real(_obj(root, "embedding", ""), "scale", "embedding.")
    entries = root.get("layers")
    if not isinstance(entries, list) or not entries or len(entries) > MAX_LAYERS:
        raise ConfigError(f"config.json: 'layers' must list 1 to {MAX_LAYERS} layers")
    norm = NormSpec("rmsnorm", width, eps)
    layers = []
    for i, entry in enumerate(entries):
        where = f"layers[{i}]."
        if not isinstance(entry, dict) or not isinstance(entry.get("type"), str):
            raise ConfigError(f"config.json: {where[:-1]} must be an object with a 'type'")
        m, w = _obj(entry, "mixer", where), where + "mixer."
        if entry["type"] == "attention":
            mixer = _attention(m, width, eps, w)
        elif entry["type"] == "retention":
            mixer = _retention(m, width, eps, w)
        else:
            raise Unsupported(f"config.json: {where[:-1]} has type {entry['type']!r}; a Lokizen layer is 'attention' or "
                              f"'retention'")
        ff = _feed_forward(_obj(entry, "mlp", where), width, where + "mlp.") if entry.get("mlp") is not None else None
        layers.append(LayerSpec(block="pre_norm", mixer=mixer, feed_forward=ff, mixer_norm=norm,
                                feed_forward_norm=norm if ff else None, weight_prefix=f"l{i}.",
                                mixer_norm_name="norm1", feed_forward_norm_name="norm2"))

    # the passes of the loop follow one another; each run of a layer has a cache entry of its own
    runs = [(i, False) for i in range(len(layers))]
    if root.get("loop") is not None:
        loop = _obj(root, "loop", "")
        start, stop = _int(loop, "start", "loop.", least=0), _int(loop, "stop", "loop.")
        times = _int(loop, "times", "loop.")
        if not start < stop <= len(layers):
            raise ConfigError(f"config.json: loop {start} .. {stop} does not lie within the {len(layers)} layers")
        if (stop - start) * times > MAX_RUNS:
            raise ConfigError(f"config.json: {times} passes over {stop - start} layers exceed {MAX_RUNS} layer runs")
        again = [(i, i == start) for i in range(start, stop)]
        runs[stop:stop] = again * (times - 1)
    return ModelSpec(architecture=ARCHITECTURE, hidden_size=width, vocab_size=vocab,
                     max_position_embeddings=MAX_POSITIONS, layers=tuple(layers),
                     run_order=tuple(RunStep(i, n, True, add_embedding=again) for n, (i, again) in enumerate(runs)),
                     final_norm=norm, tie_word_embeddings=False, eos_token_ids=(), embed_name="embed",
                     final_norm_name="final.norm", head_name="head", embed_scale=scale)
