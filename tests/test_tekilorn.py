"""Tekilorn on the host: the reader and its refusals, the program of layer calls, tensor names and shapes, cache needs, the
pages of kept first tokens, and the plain implementation against closed forms and against itself."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_tekilorn as pt
import tekilorn_helpers as th

ALL = [th.SMALL_A, th.SMALL_B, th.SMALL_C, th.SMALL_D, th.SMALL_E]


def build(doc):
    from sglang_rs_b200 import models  # noqa: F401
    from sglang_rs_b200.config import RawConfig, resolve_architecture
    raw = RawConfig.from_dict(copy.deepcopy(doc))
    entry = resolve_architecture(raw)
    config = entry.parse_config(raw)
    return config, entry.build_model(config)


def random_weights(doc, seed):
    from sglang_rs_b200.weights.random_init import random_tensors
    _, model = build(doc)
    tensors = th.spread(random_tensors(model.tensor_specs(), seed), seed)
    return {k: v.to(torch.float64).numpy() for k, v in tensors.items()}


@pytest.mark.parametrize("doc", ALL, ids="abcde")
def test_the_reader_takes_every_size_from_the_document(doc):
    config, model = build(doc)
    assert config.width == doc["width"] and config.vocab == doc["vocab"] and len(config.layers) == len(doc["layers"])
    specs = model.tensor_specs()
    assert specs["head"].shape == specs["embed"].shape == (doc["vocab"], doc["width"])
    assert ("loop.step" in specs) == ("loop" in doc)
    if "loop" in doc:
        assert specs["loop.step"].shape == (doc["loop"]["times"], doc["width"])
    for index, entry in enumerate(doc["layers"]):
        m, p = entry["mixer"], f"l{index}.mix."
        maps = 2 if entry["type"] == "attention" else 1
        assert specs[p + "q"].shape == (m["heads"] * maps * m["dim"], doc["width"])
        assert specs[p + "k"].shape == (m["kv_heads"] * maps * m["dim"], doc["width"])
        assert specs[p + "v"].shape == (m["kv_heads"] * m["vdim"], doc["width"])
        assert specs[p + "o"].shape == (doc["width"], m["heads"] * m["vdim"])
        assert (p + "g" in specs) == (maps == 1)
        for name in ("lq1", "lk1", "lq2", "lk2"):
            assert (p + name in specs) == (maps == 2)
            assert maps == 1 or specs[p + name].shape == (m["dim"],)
        f = entry["mlp"]
        if f is None:
            assert f"l{index}.norm2" not in specs
        elif f["kind"] == "moe":
            assert specs[f"l{index}.mlp.router"].shape == (f["router"]["experts"], doc["width"])
            assert f"l{index}.mlp.e{f['router']['experts']}.up" not in specs
            assert (f"l{index}.mlp.shared.up" in specs) == bool(f.get("shared")) == (f"l{index}.mlp.shared.sg" in specs)


def test_the_program_walks_the_stretch_and_opens_every_pass():
    _, model = build(th.SMALL_A)
    assert [(c.layer, c.entry, c.pass_index) for c in model.program] == [
        (0, None, 0), (1, 0, 0), (2, None, 0), (1, 0, 1), (2, None, 1), (1, 0, 2), (2, None, 2), (3, None, 0)]
    assert pt.layer_runs(th.SMALL_A) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    needs = model.cache_needs()
    assert len(needs) == 8 and needs[1] == needs[3] and needs[1] is not needs[0]
    assert (needs[0].window, needs[0].keep_first, needs[0].value_dim) == (24, 5, 8)
    assert (needs[2].window, needs[2].keep_first) == (40, 19)
    assert (needs[1].window, needs[1].keep_first, needs[1].head_dim, needs[1].value_dim) == (None, 0, 24, 20)
    _, once = build(th.SMALL_E)
    assert [(c.layer, c.entry, c.pass_index) for c in once.program] == [(0, 0, 0), (1, None, 0)]
    _, none = build(th.SMALL_B)
    assert none.pass_entries == [] and [c.layer for c in none.program] == [0, 1, 2]


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].__setitem__("type", "convolution"), "not a mixer"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("kv_heads", 3), "multiple"),
    (lambda d: d["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), "even"),
    (lambda d: d["layers"][0]["mixer"]["mask"].__setitem__("keep_first", -1), "keep_first"),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 9), "exceeds"),
    (lambda d: d["layers"][1]["mlp"].__setitem__("kind", "conv"), "not a feed-forward"),
    (lambda d: d["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("softcap", 0), "softcap"),
    (lambda d: d["layers"][1]["mixer"]["q_temp"].__setitem__("every", 0), "every"),
    (lambda d: d["loop"].__setitem__("stop", 9), "stretch"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_the_reader_refuses_what_it_cannot_build(change, message):
    from sglang_rs_b200.config import ConfigError
    doc = copy.deepcopy(th.SMALL_A)
    change(doc)
    with pytest.raises(ConfigError, match=message):
        build(doc)


def test_two_maps_and_kept_tokens_refuse_what_is_not_built_beside_them():
    from sglang_rs_b200.parts import AttentionNames, DifferentialMaps, GroupedQueryAttention, NoPositionEncoding, PagedKV, RotaryEncoding
    names = dict(q="q", k="k", v="v", o="o")
    maps = DifferentialMaps(0.5, 1e-5, "a", "b", "c", "d")
    with pytest.raises(ValueError, match="two maps"):
        GroupedQueryAttention(8, 2, 1, 8, 1.0, NoPositionEncoding(), AttentionNames(gate="g", **names), maps=maps)
    with pytest.raises(ValueError, match="two maps"):
        GroupedQueryAttention(8, 2, 1, 8, 1.0, RotaryEncoding(8, 10.0), AttentionNames(**names), maps=maps)
    with pytest.raises(ValueError, match="kept behind a window"):
        GroupedQueryAttention(8, 2, 1, 8, 1.0, NoPositionEncoding(), AttentionNames(**names), keep_first=3)
    with pytest.raises(ValueError, match="kept behind a window"):
        PagedKV(1, 8, None, keep_first=2)


@pytest.mark.parametrize("page,window,keep", [(4, 6, 3), (4, 6, 4), (4, 6, 5), (8, 3, 20), (16, 1, 1), (4, 9, 0)])
def test_pages_of_kept_tokens_stay_and_the_others_behind_the_window_go_back(page, window, keep):
    from sglang_rs_b200.cache import CacheManager
    from sglang_rs_b200.parts import PagedKV
    manager = CacheManager([PagedKV(1, 8, window, keep_first=keep)], page_size=page, max_tokens=100, max_requests=2)
    (key,) = manager.allocators
    assert key == (("kv", window, keep) if keep else ("kv", window)) and not manager.prefix_reuse_possible()
    handle = manager.open("a")
    for length in range(1, 90):
        manager.reserve(handle, 1)
        manager.commit(handle, 1)
        table = manager.allocators[key], handle.table(key)
        for logical, held in enumerate(table[1]):
            # a page is wanted while some later row (the next is at `length`) sees one of its tokens
            seen = any(pt.visible(length, j, window, keep) for j in range(logical * page, min((logical + 1) * page, length)))
            assert not seen or held >= 0, (length, logical, "a page that is still seen was given back")
            kept = logical * page < keep
            passed = (logical + 1) * page <= length - window + 1
            assert (held >= 0) == (kept or not passed), (length, logical)
        manager.check_invariants()
    manager.close(handle)
    assert manager.allocators[key].free_count == manager.allocators[key].num_pages


def test_the_pieces_of_keys_that_a_decoded_row_walks():
    from sglang_rs_b200.engine.runner import visible_pieces
    positions = np.arange(0, 400)
    for window, keep, size in ((None, 0, 32), (40, 0, 32), (41, 7, 32), (33, 70, 32), (1, 3, 64), (500, 9, 128), (64, 64, 64)):
        pieces, keys = visible_pieces(positions, window, keep, size)
        for p in positions:
            seen = [j for j in range(p + 1) if pt.visible(p, j, window, keep)]
            assert pieces[p] == len({j // size for j in seen}), (window, keep, size, p)
            assert keys[p] == len(seen)


def test_the_plain_mechanisms_against_closed_forms():
    # the pair (u, v) of an interleaved rotation turns as a complex number does; lengths stay
    x = np.random.default_rng(0).normal(size=(5, 2, 8))
    y = pt.rotate_pairs(x, np.arange(5), {"base": 100.0, "dims": 6})
    z = (x[3, 0, 2] + 1j * x[3, 0, 3]) * np.exp(1j * 3 * 100.0 ** (-2 / 6))
    assert y[3, 0, 2] == pytest.approx(z.real) and y[3, 0, 3] == pytest.approx(z.imag)
    assert np.allclose(y[0], x[0]) and np.allclose(y[..., 6:], x[..., 6:])
    # the temperature is 1 up to position every - 2 and steps at every - 1
    t = pt.query_temperature([0, 6, 7, 8, 14, 15], {"coef": 0.5, "every": 8})
    assert np.allclose(t, [1, 1, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)])
    # a window of two that keeps one: the fourth row sees rows 0, 2, 3
    q, k = np.zeros((4, 1, 2)), np.zeros((4, 1, 2))
    v = np.array([10.0, 1000.0, 20.0, 60.0]).reshape(4, 1, 1)
    assert pt.attend(q, k, v, 1.0, 2, 1)[3, 0, 0] == pytest.approx(30.0)
    # a cap: scores of +-infinity become +-cap
    q, k = np.full((2, 1, 1), 1e6), np.array([-1.0, 1.0]).reshape(2, 1, 1)
    v = np.array([1.0, 0.0]).reshape(2, 1, 1)
    assert pt.attend(q, k, v, 1.0, softcap=2.0)[1, 0, 0] == pytest.approx(math.exp(-4) / (1 + math.exp(-4)))
    # equal maps: the head's result is the normed values' mix, whatever lambda (below one)
    a = np.random.default_rng(1).normal(size=(3, 2, 6))
    assert np.allclose(pt.combine_maps(a, a, 0.4, 0.3, 0.0), 0.7 * pt.rms(a, 0.0))
    # limits: far outside, the activation is limit sigmoid(1.702 limit) (1 - limit) and so on
    w = {"gate": np.array([[1.0]]), "up": np.array([[1.0]]), "down": np.array([[1.0]])}
    assert pt.clamped(np.array([[100.0]]), w, "", 2.0)[0, 0] == pytest.approx(2.0 / (1 + math.exp(-3.404)) * 3.0)
    assert pt.clamped(np.array([[-100.0]]), w, "", 2.0)[0, 0] == pytest.approx(0.0, abs=1e-60)


def test_the_weight_is_on_the_experts_input():
    f = {"router": {"experts": 2, "top": 1}, "expert": {"limit": 50.0}}
    w = {"p.router": np.array([[0.0], [-1.0]])}
    for e in (0, 1):
        w.update({f"p.e{e}.gate": np.array([[2.0]]), f"p.e{e}.up": np.array([[3.0]]), f"p.e{e}.down": np.array([[1.0]])})
    h = np.array([[4.0]])
    g, u = 0.5 * 8.0, 0.5 * 12.0                                   # sigmoid(0) = 1/2 times the input
    assert pt.routed(h, w, "p.", f)[0, 0] == pytest.approx(g * pt.sigmoid(1.702 * g) * (u + 1))


@pytest.mark.parametrize("doc", ALL, ids="abcde")
def test_prefix_rows_do_not_depend_on_what_follows(doc):
    """The plain implementation is causal: the logits of a prefix equal the first rows of the longer run."""
    w = random_weights(doc, 3)
    tokens = th.random_requests(doc, (45,), seed=1)["r0"]
    collect = []
    whole = pt.forward(doc, w, tokens, collect)
    assert len(collect) == len(pt.layer_runs(doc)) and np.isfinite(whole).all()
    assert np.allclose(pt.forward(doc, w, tokens[:19]), whole[:19], atol=1e-9)


@pytest.mark.parametrize("wide", [False, True])
@pytest.mark.parametrize("mixer,window,keep", [("attention_2", 12, 4), ("attention", None, 0)])
def test_a_marked_key_decides_the_logits_of_the_made_models(tmp_path, mixer, window, keep, wide):
    """The models of ``tekilorn_helpers.marked_folder`` do what the GPU tests rely on: a row's logits hang on the marked key
    while it is visible (a kept first token always is), and not at all once it is out."""
    folder = th.marked_folder(tmp_path, torch.float32, mixer, window, keep, wide)
    doc, w = th.load_folder(folder)
    for mark in (3, 4, 9):
        marked, plain = th.with_mark(doc, 60, mark, seed=2)
        a, b = pt.forward(doc, w, marked), pt.forward(doc, w, plain)
        moved = np.abs(a - b).max(axis=1) / np.abs(a).max()
        assert np.all(moved[:mark] == 0.0) and moved[mark + 1] > 0.3
        if window is None or mark < keep:
            assert np.all(moved[mark + 1:] > 0.15) and moved[-1] > 0.3
        else:
            assert moved[mark + window - 1] > 0.15 and np.all(moved[mark + window:] == 0.0)
