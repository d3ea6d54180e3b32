"""The Mapovik config reader: keys, run order and passes of looped layers, declared tensors with sizes that only the tensor
knows, cache needs, refusals; tables of integers.  No GPU."""
import copy

import pytest
import torch

import plain_mapovik as P
from safetyraise_lmengine_b200 import spec_from_config
from safetyraise_lmengine_b200.errors import ConfigError, Unsupported, WeightError
from safetyraise_lmengine_b200.parts.channel_delta import block_diagonal
from safetyraise_lmengine_b200.parts.model import cache_groups_of, tensor_decls
from safetyraise_lmengine_b200.parts.position import rescaled_frequencies
from safetyraise_lmengine_b200.weights.loader import INT_TABLE, TensorDecl, check_against, load_tensors
from safetyraise_lmengine_b200.weights.random_init import RandomWeights, random_tensor

LEFT = {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 20, "scale": 0.3,
        "rot": {"base": 500.0, "dims": 8, "scaling": {"factor": 2.5}}}
RIGHT = {"heads": 6, "vdim": 10, "state": 9, "groups": 2, "norm_groups": 4, "conv": 3}
DELTA = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 14, "conv": 5}
MOE = {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2}}
CFG = {"architecture": "Mapovik", "width": 48, "vocab": 100, "norm": {"eps": 1e-4}, "residual_mult": 0.7, "logit_scale": 3.0,
       "layers": [{"type": "parallel", "mixer": {"left": LEFT, "right": RIGHT}, "mlp": MOE},
                  {"type": "channel_delta", "mixer": DELTA, "mlp": None},
                  {"type": "channel_delta", "mixer": DELTA, "mlp": {"kind": "dense", "ff": 36}}],
       "loop": {"start": 0, "stop": 2, "times": 3}}


def test_layers_and_constants():
    spec = spec_from_config(CFG)
    assert (spec.architecture, spec.hidden_size, spec.vocab_size, spec.logit_scale, spec.embed_scale) == \
        ("Mapovik", 48, 100, 3.0, 1.0)
    assert not spec.tie_word_embeddings and spec.head_name == "head" and spec.embed_norm is None
    assert (spec.final_norm.kind, spec.final_norm.eps, spec.final_norm.unit_offset) == ("layernorm", 1e-4, False)
    assert all(l.block == "pre_norm" and l.mixer_norm.kind == "layernorm" and l.sublayer_scale == 0.7 for l in spec.layers)
    side, delta = spec.layers[0].mixer, spec.layers[1].mixer
    assert (side.kind, side.combine, side.out_norm_eps) == ("side_by_side", "normed_mean", 1e-4)
    a, s = side.mixers
    assert (a.kind, a.heads, a.kv_heads, a.head_dim, a.v_head_dim, a.softmax_scale, a.window, a.softcap, a.bias) == \
        ("rotated_attention", 6, 3, 12, 20, 0.3, None, None, False)
    assert (a.position.kind, a.position.theta, a.position.rotary_dim, a.position.head_dim, a.position.divisor,
            a.position.scaling) == ("rotary_half", 500.0, 8, 12, 2.5, None)
    assert (s.kind, s.heads, s.head_dim, s.state, s.groups, s.norm_parts, s.conv_taps, s.norm_eps) == \
        ("state_space", 6, 10, 9, 2, 4, 3, 1e-4)
    assert (delta.kind, delta.heads, delta.kv_heads, delta.head_dim, delta.v_head_dim, delta.conv_taps, delta.norm_eps,
            delta.unit_eps) == ("channel_delta", 4, 2, 8, 14, 5, 1e-4, 1e-6)
    ff = spec.layers[0].feed_forward
    assert (ff.kind, ff.experts, ff.top, ff.intermediate_size, ff.activation, ff.scoring, ff.gated, ff.vocab, ff.shared_size,
            ff.weight_on_input) == ("routed_experts", 5, 2, 24, "silu", "table", True, 100, 0, False)
    dense = spec.layers[2].feed_forward
    assert (dense.kind, dense.intermediate_size, dense.activation) == ("dense", 36, "relu_squared")
    assert spec.layers[1].feed_forward is None and spec.layers[1].feed_forward_norm is None


@pytest.mark.parametrize("loop", [None, {"start": 0, "stop": 2, "times": 3}, {"start": 1, "stop": 2, "times": 2},
                                  {"start": 0, "stop": 3, "times": 2}, {"start": 2, "stop": 3, "times": 4},
                                  {"start": 1, "stop": 3, "times": 1}])
def test_looped_layers_run_in_passes_with_entries_of_their_own(loop):
    cfg = copy.deepcopy(CFG)
    cfg["loop"] = loop
    if loop is None:
        del cfg["loop"]
    spec = spec_from_config(cfg)
    assert [(s.layer, s.begins_pass) for s in spec.run_order] == P.layer_runs(cfg)
    assert all(s.writes_cache and not s.add_embedding for s in spec.run_order)
    entries = [e for s in spec.run_order for e in (s.cache,) + s.more_caches]
    assert entries == list(range(len(entries)))
    assert all(len(s.more_caches) == (1 if spec.layers[s.layer].mixer.kind == "side_by_side" else 0) for s in spec.run_order)
    assert spec.num_passes == (loop["times"] if loop else 0)
    names = {d.name: tuple(d.shape) for d in tensor_decls(spec)}
    if loop:            # one pass begins with the product and its vector, too
        assert names["loop.in"] == (48, 96) and names["loop.step"] == (loop["times"], 48)
    else:
        assert "loop.in" not in names and "loop.step" not in names


def test_declared_tensors_and_the_sizes_that_only_the_tensor_knows():
    decls = tensor_decls(spec_from_config(CFG))
    names = {d.name: tuple(d.shape) for d in decls}
    assert names["embed"] == names["head"] == (100, 48) and names["final.norm"] == (48,)
    assert names["l0.mix.left.q"] == (72, 48) and names["l0.mix.left.k"] == (36, 48) and names["l0.mix.left.v"] == (60, 48)
    assert names["l0.mix.left.o"] == (48, 120) and names["l0.mix.left.out"] == names["l0.mix.right.out"] == (48,)
    assert not any(n.startswith("l0.mix.left") and n.endswith(".b") for n in names)
    assert names["l0.mix.right.in"] == (2 * 60 + 2 * 2 * 9 + 6, 48) and names["l0.mix.right.o"] == (48, 60)
    assert names["l0.mix.right.conv"] == (96, 3) and names["l0.mix.right.conv.b"] == (96,)
    assert names["l0.mix.right.dt_bias"] == names["l0.mix.right.A_log"] == names["l0.mix.right.D"] == (6,)
    assert names["l0.mix.right.norm"] == (60,)
    assert names["l1.mix.q"] == names["l1.mix.k"] == (16, 48) and names["l1.mix.v"] == (56, 48) and names["l1.mix.b"] == (4, 48)
    assert names["l1.mix.q.conv"] == (16, 5) and names["l1.mix.v.conv"] == (56, 5)
    assert names["l1.mix.A_log"] == (4,) and names["l1.mix.dt_bias"] == (32,) and names["l1.mix.norm"] == (14,)
    assert names["l1.mix.a1"] == names["l1.mix.g1"] == (None, 48)
    assert names["l1.mix.a2"] == (32, None) and names["l1.mix.g2"] == (56, None) and names["l1.mix.o"] == (48, 56)
    assert names["l0.mlp.table"] == (100, 2) and "l0.mlp.router" not in names and names["l0.mlp.e4.gate"] == (24, 48)
    assert names["l2.mlp.up"] == (36, 48) and names["l2.mlp.down"] == (48, 36) and "l1.norm2" not in names
    have = {n: tuple(7 if d is None else d for d in s) for n, s in names.items()}
    check_against(decls, have)                                   # any rank
    with pytest.raises(WeightError, match="l2.mix.a1"):
        check_against(decls, dict(have, **{"l2.mix.a1": (7, 47)}))
    table = [d for d in decls if d.name == "l0.mlp.table"][0]
    assert (table.role, table.below, table.distinct) == (INT_TABLE, 5, True)
    made = RandomWeights(decls, seed=1).get("l0.mlp.table")
    assert made.dtype == torch.int32 and int(made.min()) >= 0 and int(made.max()) < 5 and bool((made[:, 0] != made[:, 1]).all())


def test_tables_of_integers_are_checked():
    decl = TensorDecl("t", (3, 2), INT_TABLE, below=4, distinct=True)

    class Source:
        def __init__(self, rows):
            self.t = torch.tensor(rows, dtype=torch.int32)

        def names(self):
            return ["t"]

        def meta(self, name):
            return self.t.dtype, tuple(self.t.shape), 0

        def get(self, name):
            return self.t

    load = lambda rows: load_tensors(Source(rows), [decl], torch.float32, "cpu")["t"]
    assert load([[0, 3], [2, 1], [1, 0]]).tolist() == [[0, 3], [2, 1], [1, 0]]
    for rows in ([[0, 4], [2, 1], [1, 0]], [[0, -1], [2, 1], [1, 0]], [[0, 1], [2, 2], [1, 0]]):
        with pytest.raises(WeightError, match="t "):
            load(rows)
    whole = random_tensor(TensorDecl("w", (40, 6), INT_TABLE, below=6, distinct=True), 3)
    assert bool((whole.sort(dim=-1).values == torch.arange(6)).all())


def test_cache_groups():
    groups = cache_groups_of(spec_from_config(CFG))
    delta = 4 * 8 * 14 + (2 * 2 * 8 + 4 * 14) * 4           # S, and the last four inputs of the channels
    space = 6 * 10 * 9 + (60 + 36) * 2
    by = {(g.kind, g.window, g.kv_heads, g.head_dim, g.value_dim, g.state_shape): g.entries for g in groups}
    assert by == {("paged_all", None, 3, 12, 20, ()): (0, 3, 6), ("fixed_state", None, 0, 0, 0, (space,)): (1, 4, 7),
                  ("fixed_state", None, 0, 0, 0, (delta,)): (2, 5, 8, 9)}
    odd = copy.deepcopy(CFG)
    odd["layers"][0]["mixer"]["right"] = dict(RIGHT, heads=1, vdim=5, state=3, groups=1, norm_groups=1, conv=2)
    shapes = {g.state_shape for g in cache_groups_of(spec_from_config(odd)) if g.kind == "fixed_state"}
    assert (28,) in shapes                                  # 15 + 11 floats, in whole fours


def test_frequencies_divided_by_one_number():
    assert rescaled_frequencies(500.0, 8, None, 2.5) == [500.0 ** (-2.0 * i / 8) / 2.5 for i in range(4)]


def test_block_diagonal():
    a, b = torch.ones(2, 3), 2 * torch.ones(3, 2)
    got = block_diagonal(a, b, 8)
    assert got.shape == (5, 8) and got[:2, :3].eq(1).all() and got[2:, 3:5].eq(2).all()
    assert got.sum() == a.sum() + b.sum()


def changed(path, value):
    cfg = copy.deepcopy(CFG)
    d = cfg
    for k in path[:-1]:
        d = d[k]
    if value is KeyError:
        del d[path[-1]]
    else:
        d[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path,value,error,match", [
    (("residual_mult",), KeyError, ConfigError, "residual_mult"),
    (("logit_scale",), "2", ConfigError, "logit_scale"),
    (("norm", "eps"), 0, ConfigError, "eps"),
    (("width",), True, ConfigError, "width"),
    (("layers",), [], ConfigError, "layers"),
    (("layers", 0, "type"), "attention", Unsupported, "attention"),
    (("layers", 0, "mixer", "left"), KeyError, ConfigError, "left"),
    (("layers", 0, "mixer", "left", "kv_heads"), 4, ConfigError, "kv_heads"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 7, ConfigError, "dims"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 14, ConfigError, "dims"),
    (("layers", 0, "mixer", "left", "rot", "scaling"), {"factor": 2.0, "low": 1.0}, Unsupported, "factor"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "factor"), 0, ConfigError, "factor"),
    (("layers", 0, "mixer", "right", "groups"), 4, ConfigError, "groups"),
    (("layers", 0, "mixer", "right", "norm_groups"), 7, ConfigError, "norm_groups"),
    (("layers", 0, "mixer", "right", "conv"), 0, ConfigError, "conv"),
    (("layers", 1, "mixer", "kv_heads"), 3, ConfigError, "kv_heads"),
    (("layers", 1, "mixer", "vdim"), KeyError, ConfigError, "vdim"),
    (("layers", 0, "mlp", "kind"), "gated", Unsupported, "gated"),
    (("layers", 0, "mlp", "router", "top"), 6, ConfigError, "top"),
    (("layers", 2, "mlp", "ff"), KeyError, ConfigError, "ff"),
    (("loop", "stop"), 4, ConfigError, "loop"),
    (("loop", "start"), 2, ConfigError, "loop"),
    (("loop", "times"), 0, ConfigError, "times"),
    (("loop", "times"), 1 << 20, ConfigError, "passes"),
])
def test_what_the_reader_refuses(path, value, error, match):
    with pytest.raises(error, match=match):
        spec_from_config(changed(path, value))


def test_a_rotation_or_its_scaling_may_be_absent():
    for path in (("layers", 0, "mixer", "left", "rot"), ("layers", 0, "mixer", "left", "rot", "scaling")):
        for value in (None, KeyError):
            a = spec_from_config(changed(path, value)).layers[0].mixer.mixers[0]
            assert a.position is None if path[-1] == "rot" else a.position.divisor == 1.0
