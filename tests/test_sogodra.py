"""Sogodra on the host: the reader and its refusals, tensor names and shapes, cache needs (a joint one included), sizes that
only the checkpoint knows, stretched wavelengths, and the plain implementation against closed forms and against itself."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_sogodra as ps
import sogodra_helpers as sh

ALL = [sh.SMALL_A, sh.SMALL_B, sh.SMALL_C, sh.SMALL_D, sh.SMALL_E, sh.SMALL_F]


def build(doc):
    from sglang_rs_b200 import models  # noqa: F401
    from sglang_rs_b200.config import RawConfig, resolve_architecture
    raw = RawConfig.from_dict(copy.deepcopy(doc))
    entry = resolve_architecture(raw)
    config = entry.parse_config(raw)
    return config, entry.build_model(config)


@pytest.mark.parametrize("doc", ALL, ids="abcdef")
def test_the_reader_takes_every_size_from_the_document(doc):
    config, model = build(doc)
    assert config.width == doc["width"] and config.vocab == doc["vocab"] and len(config.layers) == len(doc["layers"])
    specs, width = model.tensor_specs(), doc["width"]
    for index, entry in enumerate(doc["layers"]):
        p, m = f"l{index}.mix.", entry["mixer"]
        if entry["type"] == "mingru":
            assert specs[p + "z"].shape == (m["width"], width) and specs[p + "o"].shape == (width, m["width"])
        else:
            d = m if entry["type"] == "delta" else m["right"]
            q = p if entry["type"] == "delta" else p + "right."
            assert specs[q + "q"].shape == (d["kv_heads"] * d["dim"], width) and specs[q + "v"].shape == (d["heads"] * d["vdim"], width)
            assert specs[q + "k.conv"].shape == (d["kv_heads"] * d["dim"], d["conv"]) and specs[q + "norm"].shape == (d["vdim"],)
            if entry["type"] == "delta":
                assert specs[q + "a"].shape == (d["heads"], width) and specs[q + "dt_bias"].shape == (d["heads"],)
            else:
                assert specs[q + "a2"].shape == (d["heads"] * d["dim"], -1) and specs[q + "dt_bias"].shape == (d["heads"] * d["dim"],)
                left = m["left"]
                assert specs[p + "left.q"].shape == (left["heads"] * left["dim"], width)
                assert specs[p + "left.v"].shape == (left["kv_heads"] * left["vdim"], width)
                assert specs[p + "left.q.norm"].shape == (left["dim"],) and specs[p + "left.sink"].shape == (left["heads"],)
        assert (f"l{index}.norm2" in specs) == (entry["mlp"] is not None)


def test_a_parallel_layer_keeps_pages_and_a_state():
    from sglang_rs_b200.cache import CacheManager
    from sglang_rs_b200.parts import JointNeed, PagedKV, RequestState
    _, model = build(sh.SMALL_A)
    needs = model.cache_needs()
    assert [type(need) for need in needs] == [RequestState, JointNeed, RequestState, RequestState, JointNeed]
    pages, state = needs[1].parts
    assert pages == PagedKV(2, 16, 24, value_dim=12)
    # two inputs of 3*8 + 3*8 + 6*10 channels, then six states of 8 x 10
    assert state.shape == (2 * (24 + 24 + 60) + 6 * 80,) and state.dtype == torch.float32
    manager = CacheManager(needs, page_size=8, max_tokens=64, max_requests=2)
    assert list(manager.allocators) == [("kv", 24), ("kv", 37)] and manager.has_state and not manager.prefix_reuse_possible()
    joint = manager.layer_caches[1]
    assert joint.parts[0].group == ("kv", 24) and joint.parts[0].writable and not joint.read_only().parts[1].writable
    handle = manager.open("a")
    manager.reserve(handle, 20)
    manager.commit(handle, 20)
    manager.close(handle)
    manager.check_invariants()


def test_sizes_that_only_the_checkpoint_knows(tmp_path):
    from sglang_rs_b200.weights import WeightLoadError, build_model, load_checkpoint, write_model_folder
    folder = sh.make_folder(tmp_path, "m", sh.SMALL_C, seed=1, dtype=torch.float32)
    model, _ = build_model(folder)
    shapes = {name: spec.shape for name, spec in model.tensor_specs().items()}
    tensors = load_checkpoint(folder, shapes)
    assert tensors["l0.mix.right.a1"].shape == (5, 36) and tensors["l0.mix.right.g2"].shape == (22, 1)
    model.load(tensors, "cpu", torch.float32)
    tensors["l0.mix.right.a2"] = torch.zeros(14, 6)               # a pair whose halves do not fit
    with pytest.raises(ValueError, match="a1 has 5 rows"):
        model.load(tensors, "cpu", torch.float32)
    t = sh.make_tensors(sh.SMALL_C, 1)
    t["l0.mix.right.a2"] = t["l0.mix.right.a2"][:13]              # the other dimension is the configuration's
    bad = sh.write_folder(str(tmp_path / "bad"), sh.SMALL_C, t, torch.float32)
    with pytest.raises(WeightLoadError, match="a2 expected"):
        load_checkpoint(bad, shapes)
    # the random-weights mode fills them in
    made = write_model_folder(str(tmp_path / "made"), sh.SMALL_A, seed=2, dtype=torch.float32)
    model, _ = build_model(made)
    model.load(load_checkpoint(made, {n: s.shape for n, s in model.tensor_specs().items()}), "cpu", torch.float32)


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].__setitem__("type", "convolution"), "not a mixer"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("kv_heads", 3), "multiple"),
    (lambda d: d["layers"][1]["mixer"]["right"].__setitem__("kv_heads", 4), "right.heads.*multiple"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 7), "even"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("low"), "scaling.low"),
    (lambda d: d["layers"][1]["mixer"]["left"]["mask"].pop("size"), "mask.size"),
    (lambda d: d["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda d: d["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("conv", 40), "16 taps"),
    (lambda d: d["layers"][0]["mlp"].__setitem__("kind", "moe"), "not a feed-forward"),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda d: d["layers"][2]["mixer"].__setitem__("width", 0), "width"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d.__setitem__("layers", []), "at least one layer"),
])
def test_the_reader_refuses_what_it_cannot_build(change, message):
    from sglang_rs_b200.config import ConfigError
    doc = copy.deepcopy(sh.SMALL_A)
    change(doc)
    with pytest.raises(ConfigError, match=message):
        build(doc)


def test_wavelengths_stretched_over_a_ramp():
    from sglang_rs_b200.parts import RampScaling, RotaryEncoding
    s = sh.RAMP
    package = RotaryEncoding(16, 500.0, rotary_dim=12, scaling=RampScaling(s["factor"], s["low"], s["high"], s["original"]))
    rates = ps.frequencies({"base": 500.0, "dims": 12, "scaling": s})
    assert np.allclose(package.inverse_frequencies().double().numpy(), rates.numpy(), rtol=1e-6)
    base = np.array([500.0 ** (-2 * i / 12) for i in range(6)])
    waves = 2 * math.pi / base
    kept, slowed = waves < 100 / 5.0, waves > 100 / 1.0
    assert kept.any() and slowed.any() and (~kept & ~slowed).any()
    assert np.allclose(rates.numpy()[kept], base[kept]) and np.allclose(rates.numpy()[slowed], base[slowed] / 6.0)
    between = ~kept & ~slowed
    assert np.all(rates.numpy()[between] < base[between]) and np.all(rates.numpy()[between] > base[between] / 6.0)
    assert package.scaling.magnitude == 1.0


def test_the_plain_mechanisms_against_closed_forms():
    F = torch.float64
    # a filter of two taps: the last column is the current token's, zeros before the start
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=F)
    assert ps.causal_conv(u, torch.tensor([[2.0, 3.0]], dtype=F)).flatten().tolist() == [3.0, 32.0, 320.0]
    assert torch.allclose(ps.unit(torch.tensor([3.0, 4.0], dtype=F)), torch.tensor([0.6, 0.8], dtype=F), atol=1e-7)
    # the delta rule with beta 1 and no decay stores what it is told: a second value under the same key replaces the first, and
    # the read-out sees the write of its own token
    key, other = torch.tensor([1.0, 0.0], dtype=F), torch.tensor([0.0, 1.0], dtype=F)
    k = torch.stack([key, other, key]).reshape(3, 1, 2)
    v = torch.tensor([5.0, 7.0, 9.0], dtype=F).reshape(3, 1, 1)
    one = torch.ones(3, 1, dtype=F)
    o, last = ps.delta_recurrence(k, k, v, one, torch.ones(3, 1, 2, dtype=F))
    assert o.flatten().tolist() == [5.0, 7.0, 9.0] and last.flatten().tolist() == [9.0, 7.0]
    # a decay of one row of the state leaves the other alone
    decay = torch.ones(3, 1, 2, dtype=F)
    decay[:, :, 0] = 0.5
    _, last = ps.delta_recurrence(k, k, v * torch.tensor([1.0, 1.0, 0.0]).reshape(3, 1, 1), one * torch.tensor([[1.0], [1.0], [0.0]]), decay)
    assert last.flatten().tolist() == [5.0 * 0.25, 7.0]
    # one key and a sink of the same score share the weight
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 1.0}
    eye = torch.eye(2, dtype=F)
    w = {"q": eye, "k": eye, "v": torch.ones(1, 2, dtype=F), "q.norm": torch.ones(2, dtype=F), "k.norm": torch.ones(2, dtype=F),
         "o": torch.ones(1, 1, dtype=F), "sink": torch.tensor([2.0], dtype=F)}
    h = torch.tensor([[1.0, 1.0]], dtype=F)
    assert float(ps.windowed_attention(h, w, m, 0.0)) == pytest.approx(2.0 / 2.0)
    # minGRU: the candidate's two branches, and a gate near one takes it whole
    w = {"z": torch.zeros(2, 2, dtype=F), "z.b": torch.full((2,), 50.0, dtype=F), "x": torch.zeros(2, 2, dtype=F),
         "x.b": torch.tensor([1.5, -1.0], dtype=F), "g": torch.zeros(2, 2, dtype=F), "o": torch.eye(2, dtype=F)}
    w["g"][:, 0] = 1.0
    out = ps.min_gru(torch.tensor([[1.0, 0.0]], dtype=F), w)
    gate = 1.0 / (1.0 + math.exp(-1.0))
    assert out.flatten().tolist() == pytest.approx([2.0 * gate, gate / (1.0 + math.exp(1.0))])
    # the feed-forward's clamps
    f = ps.feed_forward(torch.tensor([[10.0]], dtype=F), {k: torch.ones(1, 1, dtype=F) for k in ("gate", "up", "down")}, {"limit": 2.0})
    assert float(f) == pytest.approx(2.0 / (1.0 + math.exp(-3.404)) * 3.0)


def test_prefix_rows_do_not_depend_on_what_follows():
    for doc in (sh.SMALL_A, sh.SMALL_C):
        tensors = sh.make_tensors(doc, 3)
        tokens = sh.random_requests(doc, (45,), seed=1)["r0"]
        whole, after = ps.forward(doc, tensors, tokens, return_layers=True)
        assert after.shape == (len(doc["layers"]), 45, doc["width"])
        assert torch.allclose(ps.forward(doc, tensors, tokens[:19]), whole[:19], atol=1e-9)


@pytest.mark.parametrize("kind,window,wide", [("window", 12, False), ("delta", None, False), ("channel", None, False), ("mingru", None, False),
                                              ("delta", None, True), ("channel", None, True)])
def test_a_mark_decides_the_logits_of_the_made_models(tmp_path, kind, window, wide):
    """The models of ``sogodra_helpers.marked_folder`` do what the GPU tests rely on."""
    folder = sh.marked_folder(tmp_path, torch.float32, kind, window, wide)
    doc, tensors = sh.load_folder(folder)
    tokens = sh.with_mark(doc, 80, 5, seed=2)
    a = ps.forward(doc, tensors, tokens).numpy()
    b = ps.forward(doc, tensors, tokens[:5] + [sh.FILL] + tokens[6:]).numpy()
    moved = np.abs(a - b).max(axis=1) / np.abs(a).max()
    assert np.all(moved[:5] == 0.0)
    if window:
        assert moved[5 + window - 1] > 0.2 and moved[5 + window] == 0.0 and moved[6] > 0.2
    else:
        assert moved[-1] > 0.2 and moved[6] > 0.2
