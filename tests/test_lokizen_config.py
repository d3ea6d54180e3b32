"""The Lokizen config reader: keys, run order of looped layers, declared tensors, cache needs, refusals; the buckets of
distances; pages of a window that keeps the first tokens.  No GPU."""
import copy
import math
import random

import pytest

import plain_lokizen as P
from safetyraise_lmengine_b200 import spec_from_config
from safetyraise_lmengine_b200.cache.manager import PAGED_WINDOW, CacheGroupSpec, CacheManager
from safetyraise_lmengine_b200.errors import ConfigError, Unsupported, WeightError
from safetyraise_lmengine_b200.parts.mixed_head_attention import distance_buckets
from safetyraise_lmengine_b200.parts.model import cache_groups_of, tensor_decls
from safetyraise_lmengine_b200.weights.loader import check_against
from safetyraise_lmengine_b200.weights.random_init import RandomWeights

ATT = {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 20, "scale": 0.3, "bias_max": 50,
       "mask": {"size": 21, "keep_first": 3}}
RET = {"heads": 2, "dim": 16, "vdim": 12, "rot": {"base": 5000.0, "dims": 8}, "decay": [0.9, 1.0]}
MOE = {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2, "scale": 1.75}}
CFG = {"architecture": "Lokizen", "width": 48, "vocab": 100, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.5},
       "layers": [{"type": "attention", "mixer": ATT, "mlp": MOE}, {"type": "retention", "mixer": RET, "mlp": None},
                  {"type": "attention", "mixer": {k: v for k, v in ATT.items() if k != "mask"}, "mlp": MOE}],
       "loop": {"start": 0, "stop": 2, "times": 3}}


def test_layers_and_constants():
    spec = spec_from_config(CFG)
    assert (spec.architecture, spec.hidden_size, spec.vocab_size, spec.embed_scale) == ("Lokizen", 48, 100, 0.5)
    assert not spec.tie_word_embeddings and spec.head_name == "head" and spec.final_norm.eps == 1e-5
    assert all(l.block == "pre_norm" and not l.mixer_norm.unit_offset for l in spec.layers)
    a, r, b = (l.mixer for l in spec.layers)
    assert (a.kind, a.heads, a.kv_heads, a.head_dim, a.v_head_dim, a.softmax_scale, a.qk_norm_eps, a.bias_max, a.window,
            a.keep_first, a.head_mix, a.output_gate) == ("mixed_head_attention", 6, 3, 12, 20, 0.3, 1e-5, 50.0, 21, 3, True, True)
    assert b.window is None and b.keep_first == 0
    assert (r.kind, r.heads, r.head_dim, r.v_head_dim, r.decay, r.norm_eps) == ("retention", 2, 16, 12, (0.9, 1.0), 1e-5)
    assert (r.position.kind, r.position.theta, r.position.rotary_dim, r.position.head_dim) == ("rotary_half", 5000.0, 8, 16)
    ff = spec.layers[0].feed_forward
    assert (ff.kind, ff.experts, ff.top, ff.intermediate_size, ff.activation, ff.scoring, ff.gated, ff.correction,
            ff.weight_scale, ff.router_bias, ff.shared_size) == \
        ("routed_experts", 5, 2, 24, "relu_squared", "logistic", False, True, 1.75, False, 0)
    assert spec.layers[1].feed_forward is None and spec.layers[1].feed_forward_norm is None


@pytest.mark.parametrize("loop", [None, {"start": 0, "stop": 2, "times": 3}, {"start": 1, "stop": 2, "times": 2},
                                  {"start": 0, "stop": 3, "times": 2}, {"start": 2, "stop": 3, "times": 4},
                                  {"start": 1, "stop": 3, "times": 1}])
def test_looped_layers_run_in_passes_with_entries_of_their_own(loop):
    cfg = copy.deepcopy(CFG)
    cfg["loop"] = loop
    if loop is None:
        del cfg["loop"]
    order = spec_from_config(cfg).run_order
    assert [(s.layer, s.add_embedding) for s in order] == P.layer_runs(cfg)
    assert [s.cache for s in order] == list(range(len(order))) and all(s.writes_cache for s in order)


def test_declared_tensors_and_the_size_that_only_the_tensor_knows():
    decls = tensor_decls(spec_from_config(CFG))
    names = {d.name: tuple(d.shape) for d in decls}
    assert names["embed"] == names["head"] == (100, 48) and names["final.norm"] == (48,)
    assert names["l0.mix.q"] == (72, 48) and names["l0.mix.k"] == (36, 48) and names["l0.mix.v"] == (60, 48)
    assert names["l0.mix.g"] == (120, 48) and names["l0.mix.o"] == (48, 120)
    assert names["l0.mix.q.norm"] == (72,) and names["l0.mix.k.norm"] == (36,)
    assert names["l0.mix.talk"] == (6, 6) and names["l0.mix.rel"] == (None, 6)
    assert names["l1.mix.q"] == names["l1.mix.k"] == (32, 48) and names["l1.mix.v"] == names["l1.mix.g"] == (24, 48)
    assert names["l1.mix.o"] == (48, 24) and "l1.norm2" not in names and "l3.norm1" not in names
    assert names["l0.mlp.router"] == (5, 48) and names["l0.mlp.correction"] == (5,) and "l0.mlp.router.b" not in names
    assert names["l2.mlp.e4.up"] == (24, 48) and names["l2.mlp.e4.down"] == (48, 24) and "l2.mlp.e0.gate" not in names
    have = {n: (14, 6) if n.endswith(".rel") else s for n, s in names.items()}
    check_against(decls, have)                                   # any number of rows
    for wrong in ((14, 5), (14,), (0, 6)):
        with pytest.raises(WeightError, match="l2.mix.rel"):
            check_against(decls, dict(have, **{"l2.mix.rel": wrong}))
    made = RandomWeights(decls, seed=1)                          # generated weights take a size of their own
    assert made.meta("l0.mix.rel")[1] == tuple(made.get("l0.mix.rel").shape) and made.meta("l0.mix.rel")[1][0] % 2 == 0


def test_cache_groups():
    groups = cache_groups_of(spec_from_config(CFG))
    by = {(g.kind, g.window, g.keep_first, g.kv_heads, g.head_dim, g.value_dim, g.state_shape): g.entries for g in groups}
    assert by == {("paged_window", 21, 3, 3, 12, 20, ()): (0, 2, 4), ("paged_all", None, 0, 3, 12, 20, ()): (6,),
                  ("fixed_state", None, 0, 0, 0, 0, (384,)): (1, 3, 5)}
    g = [g for g in groups if g.kind == "paged_window"][0]
    import torch
    assert g.bytes_per_request(torch.float32, 1000, 4) == 3 * 3 * (12 + 20) * 4 * (4 + 21 + 4 + 3) // 4 * 4


@pytest.mark.parametrize("rows,farthest", [(32, 120), (8, 64), (4, 9), (2, 7), (16, 512), (6, 81), (64, 1000), (10, 33.5)])
def test_buckets_of_distances(rows, farthest):
    got = distance_buckets(rows, farthest)
    assert len(got) == math.ceil(farthest) + 1
    assert got == [P.bucket(n, rows, farthest) for n in range(len(got))]
    assert got[:rows // 2] == list(range(rows // 2)) and got[-1] == rows - 1
    assert all(P.bucket(n, rows, farthest) == rows - 1 for n in range(len(got), 3 * len(got)))


def test_bucket_borders_that_are_whole_numbers():
    # 8 rows up to 64: h = 4, ratio 16, so bucket 4 + k begins at 4 * 2^k exactly; 6 rows up to 81: at 3 * 3^k
    assert [distance_buckets(8, 64)[n] for n in (4, 7, 8, 15, 16, 31, 32, 63, 64)] == [4, 4, 5, 5, 6, 6, 7, 7, 7]
    assert [distance_buckets(6, 81)[n] for n in (3, 8, 9, 26, 27, 80, 81)] == [3, 3, 4, 4, 5, 5, 5]


@pytest.mark.parametrize("rows,farthest,error", [(7, 50, WeightError), (0, 50, WeightError), (8, 4, ConfigError), (8, 3, ConfigError)])
def test_buckets_that_cannot_be(rows, farthest, error):
    with pytest.raises(error):
        distance_buckets(rows, farthest)


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="delta"), Unsupported),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), Unsupported),
    (lambda c: c["layers"][0]["mixer"].update(heads=4), ConfigError),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), ConfigError),
    (lambda c: c["layers"][0]["mixer"].pop("bias_max"), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), ConfigError),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.9]), ConfigError),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.9, 1.5]), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), ConfigError),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=6), ConfigError),
    (lambda c: c["layers"][2]["mlp"]["router"].pop("scale"), ConfigError),
    (lambda c: c["loop"].update(stop=4), ConfigError),
    (lambda c: c["loop"].update(start=2), ConfigError),
    (lambda c: c["loop"].update(times=0), ConfigError),
    (lambda c: c.pop("embedding"), ConfigError),
    (lambda c: c.pop("norm"), ConfigError),
    (lambda c: c.update(layers=[]), ConfigError),
])
def test_refusals(change, error):
    cfg = copy.deepcopy(CFG)
    change(cfg)
    with pytest.raises(error):
        spec_from_config(cfg)


# ---- pages of a window that keeps the first tokens ------------------------------------------------------------

KEEP = CacheGroupSpec("keep", PAGED_WINDOW, (0,), kv_heads=1, head_dim=8, window=10, keep_first=5)


def test_pages_of_the_first_tokens_stay():
    m = CacheManager([KEEP], page_size=4, num_pages=12, max_requests=2)
    s = m.open_request()
    for n in (6, 14, 30, 31, 45):
        assert m.reserve(s, n)
        m.commit(s, n)
    # 5 kept tokens lie in pages 0 and 1; after 45 tokens the next query sees keys from 36 on: page 9
    table = m.table("keep", s)
    assert [p >= 0 for p in table] == [True, True] + [False] * 7 + [True] * 3
    assert m.free_pages("keep") == 12 - 5 and m.audit() == 0
    m.truncate(s, 45)
    with pytest.raises(ValueError):
        m.truncate(s, 44 - 10)                    # its window would need pages that are gone
    m.close_request(s)
    assert m.free_pages("keep") == 12 and m.audit() == 0


def test_a_failed_step_gives_back_only_its_own_pages():
    m = CacheManager([KEEP], page_size=4, num_pages=12, max_requests=2)
    s = m.open_request()
    assert m.reserve(s, 30)
    m.commit(s, 30)
    before = m.table("keep", s)
    assert m.reserve(s, 39)
    m.truncate(s, 30)
    assert m.table("keep", s) == before and m.length(s) == 30 and m.audit() == 0


@pytest.mark.parametrize("seed", range(4))
def test_random_lives_with_kept_tokens(seed):
    rng = random.Random(seed)
    g = CacheGroupSpec("g", PAGED_WINDOW, (0,), kv_heads=1, head_dim=8, window=rng.choice((1, 3, 8, 17)),
                       keep_first=rng.choice((0, 1, 4, 9, 40)))
    m = CacheManager([g], page_size=4, num_pages=40, max_requests=3)
    live = {}
    for _ in range(400):
        if len(live) < 3 and rng.random() < 0.2:
            live[m.open_request()] = 0
        if not live:
            continue
        s = rng.choice(list(live))
        if rng.random() < 0.1:
            m.close_request(s)
            del live[s]
        else:
            n = live[s] + rng.randint(1, 9)
            if m.reserve(s, n):
                if rng.random() < 0.15:
                    m.truncate(s, live[s])
                else:
                    m.commit(s, n)
                    live[s] = n
        assert m.audit() == 0
        for t, n in live.items():
            table = m.table("g", t)
            need = set(range(max(0, n - g.window + 1), n)) | set(range(min(n, g.keep_first)))
            assert all(table[j // 4] >= 0 for j in need), (n, g.window, g.keep_first, table)
    for s in live:
        m.close_request(s)
    assert m.free_pages("g") == 40 and m.audit() == 0
