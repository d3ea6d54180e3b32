"""Lokizen in the engine against the plain implementation (tests/plain_lokizen.py): every mechanism alone and the layers
stacked and looped, under every way of cutting the work, with pages and slots used again, and through the generation
loop.  The configurations are made here; weights are random, then sharpened so that a key at a window's edge, a kept first
token, a bucket of distances, the heads' mixture, a faded state or an expert's choice shows in the result."""
import copy
import json
import math
import os

import numpy as np
import pytest
import torch
from helpers import TOL, cut_bulk_tail, cut_portions, cut_whole, note_error, random_tokens, replay

import plain_lokizen as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def attn(heads=4, kv_heads=2, dim=16, vdim=24, window=24, keep=3, bias_max=40, mlp=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "bias_max": bias_max}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def ret(heads=3, dim=16, vdim=24, dims=8, base=800.0, decay=None, mlp=None):
    decay = decay or [1.0 - 2.0 ** (-2.0 - 1.5 * h) for h in range(heads)]
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
    return {"type": "retention", "mixer": m, "mlp": mlp}


def moe(experts=6, top=2, ff=24, scale=1.3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def config(layers, width=64, vocab=200, eps=1e-6, scale=1.5, loop=None, rows=12):
    cfg = {"architecture": "Lokizen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "embedding": {"scale": scale}}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg, rows                               # rows: of every bias table (only the tensor says)


CONFIGS = {
    # each mixer alone, without and with a feed-forward behind it
    "attention": config([attn()]),
    "retention": config([ret()]),
    "experts": config([ret(heads=2, dim=8, vdim=16, dims=4, mlp=moe(experts=7, top=3, ff=40, scale=0.7))], rows=4),
    # stacked and looped: the first layer in the loop, layers of both kinds, a layer without a window, one with more kept
    # tokens than its window is long, one that keeps none
    "looped": config([attn(mlp=moe()), ret(mlp=moe()), attn(heads=2, kv_heads=2, dim=8, vdim=8, window=7, keep=19, bias_max=9),
                      ret(heads=2, dim=32, vdim=8, dims=32, mlp=moe(experts=3, top=1)),
                      attn(heads=6, kv_heads=1, dim=16, vdim=16, window=None, mlp=moe()),
                      attn(heads=4, kv_heads=4, dim=16, vdim=32, window=33, keep=0, mlp=moe(experts=4, top=4))],
                     loop=(0, 3, 3), scale=0.8),
    "loop of the last layer": config([ret(), attn(window=20, keep=1)], loop=(1, 2, 2), rows=8, scale=2.5),
    # sizes with exact tensor-core kernels: 16 heads of 64 and of 128, 32 heads; windows that end inside a tile of keys
    "wide": config([attn(heads=16, kv_heads=4, dim=64, vdim=64, window=75, keep=5, bias_max=100),
                    ret(heads=2, dim=64, vdim=64, dims=32),
                    attn(heads=16, kv_heads=2, dim=128, vdim=128, window=150, keep=40, bias_max=77, mlp=moe(experts=8, top=2, ff=32))],
                   width=128, vocab=260, rows=16),
    "many heads": config([attn(heads=32, kv_heads=4, dim=64, vdim=64, window=50, keep=33),
                          attn(heads=18, kv_heads=3, dim=32, vdim=48, window=90, keep=2, mlp=moe(experts=4, top=2, ff=16)),
                          ret(heads=1, dim=128, vdim=128, dims=128, decay=[0.99])], width=96, rows=10),
    # sizes that are 1, odd or no multiple of 8; a window of one token, a window longer than any request; decays 0 and 1
    "odd": config([attn(heads=3, kv_heads=1, dim=20, vdim=7, window=1, keep=1, bias_max=5, mlp=moe(experts=3, top=3, ff=20)),
                   attn(heads=1, kv_heads=1, dim=9, vdim=33, window=5000, keep=4, bias_max=33.5),
                   ret(heads=3, dim=10, vdim=9, dims=6, decay=[0.0, 1.0, 0.5], mlp=moe(experts=2, top=1, ff=9)),
                   ret(heads=1, dim=5, vdim=140, dims=0, decay=[0.97])], width=36, vocab=131, eps=1e-5, rows=2, loop=(2, 3, 2)),
}


def sharpen(tensors, cfg, rows, seed):
    """Random N(0, 0.02) matrices hide faults: biases of 0.02 tell no bucket from another, a mixture near zero silences
    the mixer, a router whose logits all lie near 0 follows its correction alone, values and outputs that are small add next
    to nothing.  Bias tables get ``rows`` rows of N(0, 1.5), mixtures are the unit matrix plus noise, corrections are spread
    out, and the rest is scaled up."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *shape: torch.randn(*shape, generator=g)
    scaled = lambda t, f: (t.float() * f).to(torch.bfloat16)
    tensors["embed"] = scaled(tensors["embed"], 25.0)
    for name in list(tensors):
        if name.endswith(".mix.rel"):
            tensors[name] = (1.5 * rnd(rows, tensors[name].shape[1])).to(torch.bfloat16)
        elif name.endswith(".mix.talk"):
            n = tensors[name].shape[0]
            t = torch.eye(n) + 0.7 * rnd(n, n) / n ** 0.5
            # one mixture in two is no bfloat16 matrix: it is stored in 32 bits and kept so
            tensors[name] = t if name.startswith("l2.") else t.to(torch.bfloat16)
        elif name.endswith((".q.norm", ".k.norm")):
            tensors[name] = (1.3 + 0.3 * rnd(tensors[name].shape[0]))
        elif name.endswith(".mlp.correction"):
            tensors[name] = 0.8 * rnd(tensors[name].shape[0])
        elif name.endswith(".mlp.router"):
            tensors[name] = scaled(tensors[name], 10.0)
        elif name.endswith((".mix.v", ".mix.o", ".mix.g")):
            tensors[name] = scaled(tensors[name], 4.0)
        elif name.endswith((".mix.q", ".mix.k")):
            tensors[name] = scaled(tensors[name], 6.0)
        elif ".mlp.e" in name:
            tensors[name] = scaled(tensors[name], 6.0)
    return tensors


def write_model(cfg, rows, seed, out):
    from safetyraise_lmengine_b200.weights.random_init import write_model_folder
    from safetyraise_lmengine_b200.weights.safetensors_io import WeightFolder, write_safetensors
    write_model_folder(cfg, seed, out)
    src = WeightFolder(out)
    tensors = sharpen({n: src.get(n).clone() for n in src.names()}, cfg, rows, seed + 1)
    del src
    write_safetensors(os.path.join(out, "model.safetensors"), tensors)
    return tensors


_folders = {}


def folder_of(name, tmp_path_factory):
    """(folder, config, weights) of a configuration, written once per session."""
    if name not in _folders:
        cfg, rows = CONFIGS[name]
        out = str(tmp_path_factory.mktemp("lokizen") / "m")
        _folders[name] = (out, cfg, write_model(cfg, rows, 170 + len(_folders), out))
    return _folders[name]


@pytest.fixture(scope="session", params=list(CONFIGS))
def model(request, tmp_path_factory):
    return (request.param,) + folder_of(request.param, tmp_path_factory)


_plain = {}


def plain(name, cfg, W, tokens):
    key = (name, tuple(tokens))
    if key not in _plain:
        _plain[key] = P.forward(cfg, W, tokens).numpy()
    return _plain[key]


def build(folder, dtype, num_pages=64, page_size=16, **kw):
    from safetyraise_lmengine_b200 import Engine
    kw.setdefault("max_context", 1024)
    kw.setdefault("max_batch_tokens", 512)
    return Engine.from_folder(folder, dtype=dtype, page_size=page_size, num_pages=num_pages, max_requests=4, **kw)


def check(got, model, requests, dtype):
    """float32: every position within the tolerance.  bfloat16: a router's choice is discrete, and rounding tips it between
    two experts at a few positions in a hundred; so one position in six may be off (one in sixteen more for every routed
    layer run behind the second, never more than one in three; none where no layer routes) and the median lies within half
    the tolerance, which grows with the root of the layer runs (it is set for two)."""
    name, _, cfg, W = model
    runs = len(P.layer_runs(cfg))
    routed = sum(bool(cfg["layers"][i]["mlp"]) for i, _ in P.layer_runs(cfg))
    for rid, tokens in requests.items():
        ref = plain(name, cfg, W, tokens)
        rows = np.stack([got[(rid, p)] for p in range(len(tokens))])
        err = np.abs(rows.astype(np.float64) - ref).max(axis=1) / np.abs(ref).max()
        tol = TOL[dtype] * (max(1.0, (runs / 2) ** 0.5) if dtype == "bfloat16" else 1.0)
        bad = np.nonzero(err > tol)[0]
        share = min(1 / 3, 1 / 6 + max(0, routed - 2) / 16)
        allowed = int(share * len(tokens)) + 2 if dtype == "bfloat16" and routed else 0
        assert dtype == "float32" or np.median(err) <= tol / 2, (name, rid, float(np.median(err)))
        assert bad.size <= allowed, (
            f"{name} request {rid}: first wrong position {bad[0]} of {len(tokens)} "
            f"(rel err {err[bad[0]]:.3e} > {tol:.1e}); wrong positions {bad[:20]}")
        label = dtype if dtype == "float32" else ("bfloat16, Lokizen: median over positions; the tolerance grows with the root "
                                                  "of the layer runs, one position in six may exceed it")
        note_error(label, float(err.max() if dtype == "float32" else np.median(err)), "lokizen " + name)


def all_pages_free(eng, n):
    return eng.cache.audit() == 0 and all(eng.cache.free_pages(g.name) == n for g in eng.cache.paged_groups)


def requests_for(cfg, lens=(1, 7, 33, 64, 100), seed=0):
    rng = np.random.default_rng(600 + seed)
    return {f"r{i}": random_tokens(rng, n, cfg["vocab"]) for i, n in enumerate(lens)}


# ---- the layers, under every cutting ---------------------------------------------------------------------------

def test_the_sharpened_models_use_what_they_have(model):
    """The tests below mean something only if each mechanism changes the logits by far more than the tolerances: the plain
    implementation with one of them altered differs."""
    name, _, cfg, W = model
    toks = requests_for(cfg, lens=(60,), seed=1)["r0"]
    ref = plain(name, cfg, W, toks)
    differs = lambda c, w: np.abs(P.forward(c, w, toks).numpy() - ref).max() > 50 * TOL["float32"] * np.abs(ref).max()
    for i, layer in enumerate(cfg["layers"]):
        mask = layer["mixer"].get("mask")
        if mask and mask["size"] < 50:
            for key, more in (("size", 1), ("keep_first", 1)):
                other = copy.deepcopy(cfg)
                other["layers"][i]["mixer"]["mask"][key] += more
                assert differs(other, W), (i, key)
        if layer["type"] == "retention":
            other = copy.deepcopy(cfg)
            other["layers"][i]["mixer"]["decay"] = [max(0.0, d - 0.01) for d in layer["mixer"]["decay"]]
            assert differs(other, W), (i, "decay")
        if layer["type"] == "attention" and layer["mixer"]["heads"] > 1:
            W2 = dict(W)
            W2[f"l{i}.mix.talk"] = torch.eye(layer["mixer"]["heads"])
            assert differs(cfg, W2), (i, "mixture")
        if layer["mlp"] and layer["mlp"]["router"]["top"] < layer["mlp"]["router"]["experts"]:
            W2 = dict(W)
            W2[f"l{i}.mlp.correction"] = torch.zeros_like(W[f"l{i}.mlp.correction"])
            assert differs(cfg, W2), (i, "correction")
    if cfg.get("loop"):
        other = copy.deepcopy(cfg)
        other["loop"]["times"] += 1
        assert differs(other, W)


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_requests_alone(model, dtype):
    eng = build(model[1], dtype)
    reqs = requests_for(model[2])
    got = {}
    for rid, toks in reqs.items():
        got.update(replay(eng, cut_whole(rid, toks)))
    check(got, model, reqs, dtype)
    assert all_pages_free(eng, 64)


def test_the_stream_after_every_layer_run(model):
    """float32: the engine's model is cut off behind its first k run steps and its stream compared with the plain one's
    (a looped layer counts each time it runs)."""
    from safetyraise_lmengine_b200 import StepEntry
    name, folder, cfg, W = model
    toks = requests_for(cfg, lens=(40,), seed=7)["r0"]
    streams = []
    P.forward(cfg, W, toks, streams)
    eng = build(folder, "float32")
    order = eng.model.spec.run_order
    assert len(order) == len(streams)
    for k in range(1, len(order) + 1):
        object.__setattr__(eng.model.spec, "run_order", order[:k])
        slot = eng.open_request()
        eng.step([StepEntry(slot, toks, [])])
        layer = cfg["layers"][order[k - 1].layer]
        pending = "moe.out" if layer["mlp"] else "mixed_attn.o" if layer["type"] == "attention" else "retention.proj_out"
        x = sum(eng.workspace.get(n, len(toks), cfg["width"], torch.float32).cpu().double() for n in ("residual", pending))
        eng.close_request(slot)
        assert (x - streams[k - 1]).abs().max() <= 2e-5 * streams[k - 1].abs().max(), (name, k)
    object.__setattr__(eng.model.spec, "run_order", order)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_then_token_by_token(model, dtype):
    """Most of a prompt in one step, the rest decoded one by one (replayed from CUDA graphs)."""
    eng = build(model[1], dtype)
    reqs = {k: v for k, v in requests_for(model[2]).items() if len(v) >= 33}
    got = {}
    for rid, toks in reqs.items():
        got.update(replay(eng, cut_bulk_tail(rid, toks, 32)))
    check(got, model, reqs, dtype)
    assert eng.graph_replays > 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_token_at_a_time_from_the_start(model, dtype):
    eng = build(model[1], dtype)
    reqs = requests_for(model[2], lens=(45,), seed=2)
    check(replay(eng, cut_bulk_tail("r0", reqs["r0"], 44)), model, reqs, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page_size", [4, 16, 12])
def test_portions_of_changing_size(model, dtype, page_size):
    """Portions down to two tokens, cut in the middle of pages, of key tiles, of windows and of the kept tokens."""
    eng = build(model[1], dtype, num_pages=40, page_size=page_size)
    reqs = {k: v for k, v in requests_for(model[2]).items() if len(v) >= 2}
    got = {}
    for rid, toks in reqs.items():
        got.update(replay(eng, cut_portions(rid, toks)))
        got.update({(rid + "b", p): row for (_, p), row in
                    replay(eng, cut_portions(rid, toks, sizes=(2, 2, 3, 2, 29, 2, 2, 35, 2))).items()})
    check(got, model, reqs, dtype)
    check(got, model, {rid + "b": toks for rid, toks in reqs.items()}, dtype)
    assert eng.cache.audit() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_and_reuse_of_pages_and_slots(model, dtype):
    """Up to four live requests: portions of some beside single tokens of others; requests end and new ones take their
    slots (states start from zero again) and pages (few pages, so the page freed last is used next)."""
    cfg = model[2]
    rng = np.random.default_rng(9)
    lens = {"a": 70, "b": 23, "c": 41, "d": 9, "e": 55, "f": 30, "g": 12}
    reqs = {k: random_tokens(rng, n, cfg["vocab"]) for k, n in lens.items()}
    fed = {k: 0 for k in reqs}

    def take(rid, n):
        lo = fed[rid]
        hi = fed[rid] = min(len(reqs[rid]), lo + n)
        return (rid, reqs[rid][lo:hi], list(range(hi - lo)))

    steps = [
        {"entries": [take("a", 20), take("b", 5)]},
        {"entries": [take("a", 1), take("b", 18), take("c", 2), take("d", 8)], "end": ["b"]},
        {"entries": [take("a", 1), take("c", 30), take("d", 1), take("e", 7)], "end": ["d"]},
        {"entries": [take("f", 30), take("a", 48), take("c", 1), take("e", 2)], "end": ["a", "f"]},
        {"entries": [take("g", 3), take("c", 8), take("e", 1)], "end": ["c"]},
        {"entries": [take("e", 1), take("g", 1)]},
        {"entries": [take("e", 44)]},                     # g is left out of a step and goes on
        {"entries": [take("g", 8)], "end": ["e", "g"]},
    ]
    assert all(fed[k] == len(reqs[k]) for k in reqs)
    eng = build(model[1], dtype, num_pages=24, page_size=8)
    check(replay(eng, steps), model, reqs, dtype)
    assert all_pages_free(eng, 24)
    if eng.cache.paged_groups:
        assert eng.cache.reuse_counts()[1] > 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(model, dtype):
    """300 tokens, the last 260 one by one: windows move on over decoded tokens and their pages turn over, the first
    tokens' pages stay."""
    reqs = requests_for(model[2], lens=(300,), seed=3)
    eng = build(model[1], dtype, num_pages=24, page_size=16)
    check(replay(eng, cut_bulk_tail("r0", reqs["r0"], 260)), model, reqs, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_in_portions(model, dtype):
    """500 tokens in portions of 48 (chunks of a state that end inside portions): the later ones stand behind hundreds of
    cached keys, most of them behind the window and their pages gone, the kept ones still there."""
    reqs = requests_for(model[2], lens=(500,), seed=6)
    eng = build(model[1], dtype, num_pages=40, page_size=16)
    check(replay(eng, cut_portions("r0", reqs["r0"], sizes=(48,))), model, reqs, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_in_one_step_beside_a_short_one(model, dtype):
    reqs = requests_for(model[2], lens=(600, 40), seed=8)
    eng = build(model[1], dtype, num_pages=72, page_size=16, max_batch_tokens=1024)
    got = replay(eng, [{"entries": [("r1", reqs["r1"], list(range(40))), ("r0", reqs["r0"], list(range(600)))],
                        "end": ["r0", "r1"]}])
    check(got, model, reqs, dtype)
    assert all_pages_free(eng, 72)


def test_cuttings_agree_in_float32(model):
    """Without a retention no float32 sum depends on the cutting or the batch: the same bits.  A retention's sums are formed
    token by token or by chunks of the portion: the same up to rounding."""
    reqs = requests_for(model[2], lens=(90, 37), seed=4)
    toks, other = reqs["r0"], reqs["r1"]
    eng = build(model[1], "float32")
    whole = replay(eng, cut_whole("r0", toks))
    others = [replay(eng, cut_bulk_tail("r0", toks, 40)), replay(eng, cut_portions("r0", toks)),
              replay(eng, [{"entries": [("x", other[:30], []), ("r0", toks[:50], list(range(50)))]},
                           {"entries": [("r0", toks[50:], list(range(40))), ("x", other[30:31], [])]}])]
    same_bits = all(l["type"] == "attention" for l in model[2]["layers"])
    big = max(np.abs(r).max() for r in whole.values())
    for got in others:
        for p in range(len(toks)):
            a, b = whole[("r0", p)], got[("r0", p)]
            assert np.array_equal(a, b) if same_bits else np.abs(a - b).max() <= TOL["float32"] * big, p


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_refused_step_leaves_nothing_behind(model, dtype):
    from safetyraise_lmengine_b200 import StepEntry
    from safetyraise_lmengine_b200.errors import ShapeError
    reqs = requests_for(model[2], lens=(30,), seed=5)
    toks = reqs["r0"]
    eng = build(model[1], dtype)
    slot = eng.open_request()
    rows = [eng.step([StepEntry(slot, toks[:11], list(range(11)))]).cpu().numpy().copy()]
    with pytest.raises(ShapeError):
        eng.step([StepEntry(slot, [model[2]["vocab"] + 5, 1], [0])])
    rows.append(eng.step([StepEntry(slot, toks[11:], list(range(19)))]).cpu().numpy().copy())
    check({("r0", p): r for p, r in enumerate(np.concatenate(rows))}, model, reqs, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_step_taken_back_restores_the_states(model, dtype):
    """launch, then revoke: states, lengths and pages as before; the request goes on as if nothing had run."""
    from safetyraise_lmengine_b200 import StepEntry
    reqs = requests_for(model[2], lens=(50,), seed=11)
    toks = reqs["r0"]
    eng = build(model[1], dtype)
    slot = eng.open_request()
    rows = [eng.step([StepEntry(slot, toks[:20], list(range(20)))]).cpu().numpy().copy()]
    prep = eng.prepare([StepEntry(slot, list(reversed(toks))[:25], [0])])
    eng.launch(prep)
    eng.revoke(prep)
    rows.append(eng.step([StepEntry(slot, toks[20:], list(range(30)))]).cpu().numpy().copy())
    check({("r0", p): r for p, r in enumerate(np.concatenate(rows))}, model, reqs, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(model, dtype):
    from safetyraise_lmengine_b200 import LLM, SamplingParams
    name, folder, cfg, W = model
    rng = np.random.default_rng(21)
    prompts = [random_tokens(rng, n, cfg["vocab"]) for n in (5, 19, 11, 3, 26)]        # more requests than slots
    llm = LLM.from_folder(folder, dtype=dtype, page_size=4, num_pages=64, max_active=3, max_batch_tokens=48,
                          prefill_chunk=8, max_context=128, queue_capacity=8)
    llm.eos = set()
    res = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=10))
    off = 0
    for prompt, r in zip(prompts, res):
        assert r.finish_reason == "length" and len(r.tokens) == 10
        ref = P.forward(cfg, W, (list(prompt) + list(r.tokens))[:-1]).numpy()
        for i, tok in enumerate(r.tokens):
            row = ref[len(prompt) - 1 + i]
            slack = 1e-5 if dtype == "float32" else 3 * TOL[dtype] * max(1.0, (len(P.layer_runs(cfg)) / 2) ** 0.5)
            off += not row[tok] >= row.max() - slack * np.abs(row).max()
    # bfloat16: a tipped router (see check) may tip a token too
    assert off <= (0 if dtype == "float32" or not any(l["mlp"] for l in cfg["layers"]) else 6), off
    assert all_pages_free(llm.engine, 64)


# ---- mechanisms alone, with inputs made so that a fault shows ---------------------------------------------------

class _Ctx:
    """The fields of a step's context that the kernels' wrappers read."""
    def __init__(self, q_lens, kv_lens, dev, slots=None):
        from safetyraise_lmengine_b200.parts import Workspace
        self.n_entries, self.max_q_len = len(q_lens), max(q_lens)
        self.cu_q = torch.tensor(np.concatenate([[0], np.cumsum(q_lens)]), dtype=torch.int32, device=dev)
        self.kv_lens = torch.tensor(kv_lens, dtype=torch.int32, device=dev)
        self.positions = torch.tensor(sum((list(range(k - q, k)) for q, k in zip(q_lens, kv_lens)), []), dtype=torch.int32, device=dev)
        self.entry_of_token = torch.tensor(sum(([e] * q for e, q in enumerate(q_lens)), []), dtype=torch.int32, device=dev)
        self.kv_bound, self.workspace = max(kv_lens), Workspace(torch.device(dev), sum(q_lens))
        self.host = {"q_lens": list(q_lens)}
        self.slots = torch.tensor(slots if slots is not None else range(len(q_lens)), dtype=torch.int32, device=dev)


def _paged(keys, page_size, order, dtype, dev, gone=()):
    """keys [L, heads, d] -> (pool [pages, heads, page_size, d], table); pages in ``gone`` are not stored and their table
    entries are -1, as a window group leaves them; what no key fills is NaN."""
    L, H, d = keys.shape
    pool = torch.full((len(order), H, page_size, d), float("nan"), dtype=dtype, device=dev)
    table = []
    for i in range(-(-L // page_size)):
        table.append(-1 if i in gone else order[i])
        if i not in gone:
            chunk = keys[i * page_size:(i + 1) * page_size]
            pool[order[i], :, :chunk.shape[0]] = chunk.transpose(0, 1).to(dtype)
    return pool, table


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dk,dv,window,keep,page", [
    (4, 2, 24, 40, 100, 5, 16), (3, 1, 20, 9, 37, 50, 8), (2, 2, 16, 16, 0, 0, 16), (12, 3, 64, 128, 129, 16, 16),
    (16, 4, 64, 64, 65, 33, 12), (16, 2, 128, 128, 150, 4, 16), (32, 4, 128, 128, 96, 31, 32), (18, 3, 48, 192, 64, 0, 4),
    (40, 8, 32, 32, 70, 3, 16)])
def test_attention_kernels_at_the_edges(dtype, heads, kv_heads, dk, dv, window, keep, page):
    """Queries aimed at one key each: just inside the window and just outside it (where a heavier key waits), the last kept
    token and the one behind it, far back, at page and tile borders, at themselves.  A window one token off, a lost kept
    token, a bias of the neighbouring distance, a head's weights left unmixed or a page that was given back and read all
    the same change the result by far more than the tolerance."""
    from safetyraise_lmengine_b200.kernels import ops
    from safetyraise_lmengine_b200.parts.mixed_head_attention import distance_buckets
    dev, L = "cuda:0", 500
    cdt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(dk * 100 + dv)
    q = 0.4 * torch.randn(L, heads, dk, generator=g)
    k, v = torch.randn(L, kv_heads, dk, generator=g), torch.randn(L, kv_heads, dv, generator=g)
    rep, w = heads // kv_heads, window or L
    scale, farthest = 0.8, 90
    aims = [(L - 1, L - w), (L - 2, L - 2 - w), (L - 3, L - 3 - w + 1), (450, keep - 1), (451, keep), (452, 452), (460, 448),
            (461, 460 // page * page), (470, 470 - 31), (200, 0)]
    for row, col in aims:
        if 0 <= col <= row:
            q[row] = 7.0 * (k[col] / k[col].norm(dim=-1, keepdim=True)).repeat_interleave(rep, 0) + 0.1 * q[row]
    if dtype == "bfloat16":
        q, k, v = (t.bfloat16().float() for t in (q, k, v))
    table = 2.0 * torch.randn(10, heads, generator=g)
    talk = torch.eye(heads) + torch.randn(heads, heads, generator=g) / heads ** 0.5
    gate = torch.randn(L, 5 + heads * dv, generator=g)
    args = (q, k, v, scale, table, farthest)
    ref = P.mixed_attention(*args, talk, window, keep)
    row = lambda *a: P.mixed_attention(*a)[L - 60:]
    tail = ref[L - 60:]
    assert (tail - row(*args, torch.eye(heads), window, keep)).abs().max() > 0.1
    if window:
        assert (tail - row(*args, talk, window + 1, keep)).abs().max() > 0.1
        assert (tail - row(*args, talk, window - 1, keep)).abs().max() > 0.1
        if 0 < keep < L - w:
            assert (tail - row(*args, talk, window, keep - 1)).abs().max() > 0.1
            assert (tail - row(*args, talk, window, keep + 1)).abs().max() > 0.1
    assert (tail - row(q, k, v, scale, table.roll(1, 0), farthest, talk, window, keep)).abs().max() > 0.1
    ref = (ref.reshape(L, heads * dv) * torch.sigmoid(gate[:, 5:].double())).numpy()
    bias = table[torch.tensor(distance_buckets(10, farthest))].t().contiguous().to(dev)
    pages = -(-L // page)
    qdt = ops.mixed_head_query_dtype(cdt, heads, kv_heads, dk, dv)
    on_tensor_cores = heads <= 32 and dk % 16 == 0 and dv % 16 == 0
    assert dtype == "float32" or (qdt == torch.bfloat16) == on_tensor_cores
    tol = 2e-5 if dtype == "float32" else 1.5e-2
    # (tokens of the step, context behind it) an entry: a prompt, decoded tokens, portions, a mixed batch
    for batch in ([(L, L)], [(1, L)], [(2, L)], [(1, L), (1, 1), (1, 470), (1, 33)], [(33, L)], [(60, 481), (1, L), (2, 2), (17, 300)]):
        kp, vp, tables = None, None, []
        for n, (ql, kl) in enumerate(batch):
            first = max(0, kl - ql - w + 1) if window else 0
            gone = [i for i in range(pages) if (i + 1) * page <= first and i * page >= keep] if window else []
            order = torch.randperm(pages, generator=g).tolist()
            a, ta = _paged(k[:kl], page, order, cdt, dev, gone)
            b, _ = _paged(v[:kl], page, order, cdt, dev, gone)
            kp, vp = (a, b) if kp is None else (torch.cat([kp, a]), torch.cat([vp, b]))
            tables.append([t if t < 0 else t + n * pages for t in ta])
        width = max(map(len, tables))
        bt = torch.tensor([t + [-1] * (width - len(t)) for t in tables], dtype=torch.int32, device=dev)
        rows = torch.cat([torch.arange(kl - ql, kl) for ql, kl in batch])
        ctx = _Ctx([ql for ql, _ in batch], [kl for _, kl in batch], dev)
        out = torch.full((len(rows), heads * dv), float("nan"), dtype=cdt, device=dev)
        for split in ((True, False) if dtype == "bfloat16" else (True,)):
            ops.split_mixed_heads = split
            try:
                ops.mixed_head_attention(ctx, q[rows].reshape(len(rows), -1).to(dev, qdt), kp, vp, out, bt, heads, kv_heads, dk, dv,
                                         scale, window, keep, bias=bias, mix=talk.to(dev), gate=(gate[rows].to(dev), 5))
            finally:
                ops.split_mixed_heads = True
            err = np.abs(out.float().cpu().numpy() - ref[rows]).max(axis=1) / np.abs(ref).max()
            assert err.max() < tol, (batch, split, int(rows[err.argmax()]), float(err.max()))


@pytest.mark.parametrize("proj_cols", [0, 9])
def test_the_norm_over_all_heads(proj_cols):
    from safetyraise_lmengine_b200.kernels import ops
    dev = "cuda:0"
    g = torch.Generator().manual_seed(4)
    for T, nq, nkv, dk, dv, page in ((5, 4, 2, 24, 16, 4), (1, 1, 1, 3, 5, 16), (33, 6, 3, 64, 40, 8)):
        proj = torch.randn(T, nq * dk + nkv * (dk + dv) + proj_cols, generator=g)
        proj[:, :dk] *= 9.0                                   # one loud head: a norm per head would hide it from the others
        qw, kw = 1 + torch.rand(nq * dk, generator=g), 1 + torch.rand(nkv * dk, generator=g)
        slots = torch.randperm(8 * page, generator=g)[:T].int()
        kp, vp = torch.zeros(8, nkv, page, dk, device=dev), torch.zeros(8, nkv, page, dv, device=dev)
        for qdt in (torch.float32, torch.bfloat16):
            q = torch.zeros(T, nq * dk, dtype=qdt, device=dev)
            ops.attention_wide_norm_append(proj.to(dev), qw.to(dev), kw.to(dev), 1e-3, q, kp, vp, slots.to(dev), nq, nkv, dk, dv)
            want_q = P.rms_norm(proj[:, :nq * dk], qw, 1e-3)
            want_k = P.rms_norm(proj[:, nq * dk:(nq + nkv) * dk], kw, 1e-3).view(T, nkv, dk)
            want_v = proj[:, (nq + nkv) * dk:(nq + nkv) * dk + nkv * dv].view(T, nkv, dv).double()
            assert (q.cpu().double() - want_q).abs().max() < (1e-5 if qdt == torch.float32 else 5e-3) * want_q.abs().max()
            for t in range(T):
                pg, off = int(slots[t]) // page, int(slots[t]) % page
                assert (kp[pg, :, off].cpu().double() - want_k[t]).abs().max() < 1e-5 * want_k.abs().max()
                assert torch.equal(vp[pg, :, off].cpu().double(), want_v[t])


@pytest.mark.parametrize("chunked", [True, False])
@pytest.mark.parametrize("H,d,dv,dims", [(4, 48, 48, 48), (3, 128, 128, 64), (2, 16, 56, 0), (5, 64, 128, 32), (1, 256, 256, 256),
                                         (2, 100, 36, 20), (2, 128, 72, 128), (3, 20, 130, 4), (2, 42, 30, 8), (2, 300, 20, 2)])
def test_retention_kernels(H, d, dv, dims, chunked):
    """From states that are not zero, in slots of any order: entries of one token, of a few, of whole and broken chunks; a
    far token that outweighs the rest under a decay near one, decays of zero and one."""
    from safetyraise_lmengine_b200.kernels import ops
    from safetyraise_lmengine_b200.parts import Rotation
    dev = "cuda:0"
    g = torch.Generator().manual_seed(H * 1000 + d)
    decay = [0.9995, 0.0, 1.0, 0.6, 0.95][:H]
    for lens in ([1], [1, 5, 2], [200], [64, 1, 65, 3, 9, 130], [12, 8, 128]):
        T, n = sum(lens), len(lens)
        proj = torch.randn(T, 2 * H * d + 2 * H * dv, generator=g)
        proj[0, H * d:2 * H * d] *= 12.0                      # the first token's key stands out
        ang = 3 * torch.randn(T, dims // 2, generator=g)
        rot = Rotation(ang.cos().to(dev), ang.sin().to(dev), dims // 2) if dims else None
        slots = torch.randperm(n + 2, generator=g)[:n].tolist()
        state = torch.randn(n + 2, H * d * dv, generator=g)
        want_state, want = state.clone().double(), []
        at = 0
        for e, ql in enumerate(lens):
            p = proj[at:at + ql].double()
            def turned(x):
                if not dims:
                    return x
                h, a = dims // 2, ang[at:at + ql].float()
                c, s = a.cos().double()[:, None], a.sin().double()[:, None]
                return torch.cat([x[..., :h] * c - x[..., h:dims] * s, x[..., h:dims] * c + x[..., :h] * s, x[..., dims:]], -1)
            q = turned(p[:, :H * d].view(ql, H, d))
            k = turned(p[:, H * d:2 * H * d].view(ql, H, d)) * d ** -0.5
            o, S = P.retention_state(q, k, p[:, 2 * H * d:2 * H * d + H * dv].view(ql, H, dv), decay,
                                     want_state[slots[e]].view(H, d, dv))
            want_state[slots[e]] = S.reshape(-1)
            want.append(P.rms_norm(o, None, 1e-5).reshape(ql, H * dv) * P.silu(p[:, 2 * H * d + H * dv:]))
            at += ql
        want = torch.cat(want)
        got_state = state.to(dev)
        out = torch.full((T, H * dv), float("nan"), device=dev)
        ops.retention_in_chunks = chunked
        try:
            ops.retention(_Ctx(lens, lens, dev, slots), proj.to(dev), rot, torch.tensor(decay, device=dev), 1e-5, got_state, out, H, d, dv)
        finally:
            ops.retention_in_chunks = True
        assert (out.cpu().double() - want).abs().max() < 2e-5 * want.abs().max(), lens
        assert (got_state.cpu().double() - want_state).abs().max() < 1e-5 * want_state.abs().max(), lens


def test_corrected_choice_and_scaled_weights():
    """The best expert by score loses to a worse one with a better correction, and the winner is weighted by its score."""
    from safetyraise_lmengine_b200.kernels import ops
    dev = "cuda:0"
    g = torch.Generator().manual_seed(6)
    for T, E, top in ((40, 5, 2), (1, 3, 3), (700, 40, 7), (3, 1, 1)):
        logits = 2 * torch.randn(T, E + 3, generator=g)
        correction = torch.randn(E, generator=g)
        s = torch.sigmoid(logits[:, 3:].double())
        idx = (s + correction.double()).topk(top, dim=-1).indices
        want = s.gather(-1, idx) * 2.5
        if E > top:
            assert (idx.sort(-1).values != s.topk(top, dim=-1).indices.sort(-1).values).any()
        d = lambda t: t.to(dev)
        choice, weight = torch.zeros(T, top, dtype=torch.int32, device=dev), torch.zeros(T, top, device=dev)
        kw = dict(scoring="logistic", correction=d(correction), weight_scale=2.5)
        ops.moe_route(d(logits), None, top, choice, weight, column=3, experts=E, **kw)
        assert torch.equal(choice.cpu().long(), idx) and (weight.cpu().double() - want).abs().max() < 1e-6
        if ops.moe_sort_routes(T, E):
            choice2, weight2 = torch.zeros_like(choice), torch.zeros_like(weight)
            i32 = lambda n: torch.zeros(n, dtype=torch.int32, device=dev)
            ops.moe_sort(choice2, E, i32(E + 1), i32(E + 1), i32(T * top), i32(T * top), route=(d(logits), 3, None, weight2), **kw)
            assert torch.equal(choice2, choice) and torch.equal(weight2, weight)


@pytest.mark.parametrize("form", ["simt", "mma", "tiles"])
def test_squared_activation_of_the_grouped_products(form):
    from safetyraise_lmengine_b200.kernels import ops
    dev, E, top, T, H, ff = "cuda:0", 3, 2, 150, 64, 48
    dtype = torch.float32 if form == "simt" else torch.bfloat16
    g = torch.Generator().manual_seed(8)
    x = torch.randn(T, H, generator=g).to(dtype)
    up = (0.4 * torch.randn(E, ff, H, generator=g)).to(dtype)
    choice = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).int()
    i32 = lambda n, v=0: torch.full((n,), v, dtype=torch.int32, device=dev)
    n = T * top
    want = torch.clamp(torch.einsum("td,efd->tef", x.double(), up.double()), min=0) ** 2
    if form == "tiles":
        tiles = n // 128 + E
        group, por, rop = i32(tiles), i32(tiles * 128), i32(n)
        ops.moe_sort(choice.to(dev), E, i32(E + 1), i32(E + 1), por, rop, tile_rows=128, group_of_tile=group)
        xs, y = torch.empty(tiles * 128, H, dtype=dtype, device=dev), torch.zeros(tiles * 128, ff, dtype=dtype, device=dev)
        ops.moe_gather_rows(x.to(dev), por, top, xs)
        ops.gemm_tn_tcgen05_grouped(xs, up.to(dev), y, group, act="relu_squared")
    else:
        offsets, tiles, por, rop = i32(E + 1), i32(E + 1), i32(n), i32(n)
        ops.moe_sort(choice.to(dev), E, offsets, tiles, por, rop)
        y = torch.zeros(n, ff, dtype=dtype, device=dev)
        ops.moe_grouped(x.to(dev), por, top, up.to(dev), y, offsets, tiles, act="relu_squared")
    got = y.cpu().double()[rop.cpu().long()].view(T, top, ff)
    ref = torch.stack([want[torch.arange(T), choice[:, c].long()] for c in range(top)], 1)
    assert (got - ref).abs().max() < (1e-5 if form == "simt" else 1e-2) * ref.abs().max()


def test_embedding_scaled_and_added_again():
    from safetyraise_lmengine_b200.kernels import ops
    dev = "cuda:0"
    table = torch.randn(9, 70).bfloat16()
    ids = torch.tensor([3, 8, 0], dtype=torch.int32)
    out, flag = torch.zeros(3, 70, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    ops.embed_gather(ids.to(dev), table.to(dev), out, flag, scale=2.5)
    want = table[ids.long()].float() * 2.5
    assert torch.equal(out.cpu(), want)
    ops.embed_gather(ids.to(dev), table.to(dev), out, flag, scale=2.5, add=True)
    assert torch.equal(out.cpu(), want + want) and int(flag) == 0


# ---- as a user runs it: the command line and the trace replay ---------------------------------------------------

def test_command_line_and_trace_replay(tmp_path, tmp_path_factory):
    import subprocess
    import sys
    from conftest import ROOT
    folder, cfg, W = folder_of("looped", tmp_path_factory)
    env = dict(os.environ, PYTHONPATH=ROOT)
    cli = lambda *a: subprocess.run([sys.executable, "-m", "safetyraise_lmengine_b200", *a], env=env,
                                    capture_output=True, text=True, timeout=600)
    out = cli("inspect", "--model-path", folder, "--context", "64")
    assert out.returncode == 0, out.stderr
    info = json.loads(out.stdout)
    assert info["spec"]["architecture"] == "Lokizen" and len(info["cache_groups"]) >= 5
    svc, req = tmp_path / "svc.json", tmp_path / "req.json"
    svc.write_text(json.dumps({"model_path": folder, "model_name": "looped",
                               "engine": {"max_context": 128, "max_active": 2, "prefill_chunk": 4, "page_size": 4,
                                          "num_pages": 40, "dtype": "float32", "max_batch_tokens": 32}}))
    prompt = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5]
    req.write_text(json.dumps({"prompt_ids": prompt, "max_tokens": 6, "temperature": 0.0}))
    out = cli("run", "--config", str(svc), "--request", str(req))
    assert out.returncode == 0, out.stderr
    res = json.loads(out.stdout)
    toks = list(prompt)
    for tok in res["tokens"]:
        row = P.forward(cfg, W, toks)[-1].numpy()
        assert row[tok] >= row.max() - 1e-5 * np.abs(row).max()
        toks.append(tok)
    assert len(res["tokens"]) == 6 and res["finish_reason"] == "length"

    rng = np.random.default_rng(2)
    a, b = random_tokens(rng, 50, cfg["vocab"]), random_tokens(rng, 40, cfg["vocab"])
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[30:32], "want": [1]}, {"id": "b", "tokens": b[:39], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "b", "tokens": b[39:], "want": [0]}, {"id": "a", "tokens": a[32:], "want": [17]}],
         "end": ["a", "b"]},
    ]
    out_dir = tmp_path / "out_float32"
    proc = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out",
                           str(out_dir), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split() == ["done", "0", "done", "1", "done", "2"]
    read = lambda i: np.fromfile(out_dir / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
    ra, rb = plain("looped", cfg, W, a), plain("looped", cfg, W, b)
    biggest = max(np.abs(ra).max(), np.abs(rb).max())
    for got, ref in ((read(0), ra[[0, 29]]), (read(1), ra[[31]]), (read(2), np.stack([rb[39], ra[49]]))):
        assert got.shape == ref.shape and np.abs(got - ref).max() <= TOL["float32"] * biggest


# ---- configurations drawn at random: layer order, sizes and constants that no other test chose -----------------

def random_config(seed):
    rng = np.random.default_rng(3000 + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    width, layers, rows = pick(40, 64, 96, 128, 160), [], pick(2, 6, 14, 20, 40)
    for i in range(int(rng.integers(2, 6))):
        mlp = None
        if rng.random() < 0.7:
            experts = pick(1, 2, 3, 5, 12)
            mlp = moe(experts=experts, top=int(rng.integers(1, min(experts, 4) + 1)), ff=pick(8, 16, 24, 40, 50), scale=pick(0.6, 1.0, 2.5))
        if rng.random() < 0.55:
            kv = pick(1, 2, 3, 5)
            dim, vdim = pick((8, 8), (16, 40), (24, 16), (32, 64), (64, 64), (128, 128), (48, 128), (80, 56), (112, 160))
            layers.append(attn(heads=kv * pick(1, 2, 4), kv_heads=kv, dim=dim, vdim=vdim, window=pick(None, 1, 9, 16, 50, 129, 1000),
                               keep=pick(0, 1, 2, 9, 40), bias_max=rows + pick(1, 30, 200), mlp=mlp, scale=pick(None, 0.1, 0.5)))
        else:
            H, dim = pick(1, 2, 3, 6), pick(8, 20, 32, 40, 64, 96)
            layers.append(ret(heads=H, dim=dim, vdim=pick(8, 16, 31, 64, 130), dims=pick(0, 2, dim // 2 // 2 * 2, dim),
                              base=pick(100.0, 10000.0, 5e5), decay=[float(v) for v in rng.uniform(0.3, 1.0, H) ** 0.1], mlp=mlp))
    n = len(layers)
    start = int(rng.integers(n))
    loop = (start, int(rng.integers(start + 1, n + 1)), int(rng.integers(1, 4))) if rng.random() < 0.7 else None
    return config(layers, width=width, vocab=pick(97, 160, 301), eps=pick(1e-6, 1e-5, 1e-4), scale=pick(0.3, 1.0, 4.0), loop=loop, rows=rows)


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Whatever the order of layers and the sizes: float32 within the tolerance at every position under a cutting with
    portions, decoded tokens and a second request beside it; bfloat16 by the rule of `check`."""
    cfg, rows = random_config(seed)
    out = str(tmp_path / "m")
    W = write_model(cfg, rows, 950 + seed, out)
    rng = np.random.default_rng(seed)
    reqs = {"a": random_tokens(rng, 180, cfg["vocab"]), "b": random_tokens(rng, 37, cfg["vocab"])}
    a, b = reqs["a"], reqs["b"]
    steps = [{"entries": [("a", a[:61], list(range(61)))]},
             {"entries": [("b", b[:2], [0, 1]), ("a", a[61:64], [0, 1, 2])]},
             {"entries": [("a", a[64:150], list(range(86))), ("b", b[2:3], [0])]},
             {"entries": [("b", b[3:36], list(range(33))), ("a", a[150:151], [0])]}]
    steps += [{"entries": [("a", a[i:i + 1], [0])] + ([("b", b[36:], [0])] if i == 151 else [])} for i in range(151, 180)]
    model = (f"random {seed}", out, cfg, W)
    for dtype in DTYPES:
        eng = build(out, dtype, num_pages=20, page_size=16)
        check(replay(eng, steps), model, reqs, dtype)
        assert all_pages_free(eng, 20)
