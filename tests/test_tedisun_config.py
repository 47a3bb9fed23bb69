"""Tedisun on the host: registry, configuration keys and errors, which cache and state every layer gets, the tensors the
model asks for, frequencies, and the plain functions against closed forms."""
import copy
import math

import numpy as np
import pytest
import torch

from lgml_b200.cache import CacheManager, FixedState, PagedKV
from lgml_b200.config import ConfigError, TedisunConfig, architectures, config_from_dict
from lgml_b200.models import build_model
from lgml_b200.models.tedisun import rotation_of
from lgml_b200.parts import frequency_factors, make_part
from tests import tedisun_helpers as L
from tests.plain import tedisun_plain as P


def test_registered_by_name():
    assert "Tedisun" in architectures()
    cfg = config_from_dict(L.MIXED)
    assert isinstance(cfg, TedisunConfig) and cfg.vocab_size == 97 and cfg.hidden_size == 72 and cfg.num_hidden_layers == 4
    assert cfg.embed_scale == 3.0 and cfg.streams == 3 and cfg.logit_softcap == 20.0
    again = config_from_dict(cfg.to_dict())
    assert again.to_dict() == cfg.to_dict()
    plain = config_from_dict(L.ODD)
    assert plain.embed_scale == 1.0 and plain.logit_softcap is None and plain.streams == 1


@pytest.mark.parametrize("edit,key", [
    (lambda d: d.pop("width"), "width"),
    (lambda d: d.pop("streams"), "streams"),
    (lambda d: d.__setitem__("streams", 9), "streams"),
    (lambda d: d["norm"].pop("eps"), "norm"),
    (lambda d: d.__setitem__("logit_softcap", "high"), "logit_softcap"),
    (lambda d: d["layers"][0].__setitem__("type", "serial"), "layers[0].type"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("conv", 0), "conv"),
    (lambda d: d["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda d: d["layers"][1]["mixer"]["left"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 34), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("low"), "low"),
    (lambda d: d["layers"][1]["mixer"]["left"]["mask"].__setitem__("size", 0), "size"),
    (lambda d: d["layers"][1]["mixer"]["left"]["mask"].__setitem__("keep_first", -1), "keep_first"),
    (lambda d: d["layers"][3]["mixer"]["right"].__setitem__("gate_cap", 0), "gate_cap"),
    (lambda d: d["layers"][0]["mlp"].__setitem__("kind", "dense"), "mlp.kind"),
    (lambda d: d["layers"][0]["mlp"]["router"].__setitem__("top", 7), "top"),
    (lambda d: d["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
])
def test_a_bad_key_is_named(edit, key):
    d = copy.deepcopy(L.MIXED)
    edit(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert key.split(".")[-1] in str(e.value)


def test_cache_and_state_of_every_layer():
    up4 = lambda n: -(-n // 4) * 4
    for cfg in L.CONFIGS.values():
        model = build_model(config_from_dict(cfg))
        layout = model.cache_layout()
        assert sorted(layout) == list(range(len(cfg["layers"]))) and model.graph_safe
        for ci, layer in enumerate(cfg["layers"]):
            m = layer["mixer"]
            if layer["type"] == "delta":
                S = m["heads"] * m["dim"] * m["vdim"]
                conv = (m["conv"] - 1) * (2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"])
                assert layout[ci] == FixedState((up4(up4(S) + conv),), torch.float32)
            else:
                l, r = m["left"], m["right"]
                mask = l.get("mask", {})
                pages, state = layout[ci]
                assert pages == PagedKV(l["kv_heads"], l["dim"], mask.get("size"), l["vdim"], keep_first=mask.get("keep_first", 0))
                assert state == FixedState((up4(r["heads"] * ((r["vdim"] + 1) * r["dim"] + 1)),), torch.float32)


def test_a_window_gives_pages_back_and_keeps_the_first_tokens():
    """Keeping 67 tokens takes two pages beside the window's."""
    model = build_model(config_from_dict(L.WIDE_HEADS))
    cm = CacheManager(model.cache_layout(), n_pages=40, max_slots=2, dtype=torch.float32, device="cpu", max_step_tokens=64)
    req = cm.open("a")
    for _ in range(12):
        assert cm.reserve(req, 50)
        cm.commit(req, 50)
    for gi, grp in enumerate(cm.groups):
        kept, size = grp.spec.keep_first, grp.spec.window
        held = [b for b, p in enumerate(req.tables[gi]) if p >= 0]
        first = (600 - size + 1) // 64
        assert held == sorted(set(range(-(-kept // 64))) | set(range(first, 10)))
    cm.check()
    cm.close(req)
    cm.check()


def test_tensors_the_model_asks_for():
    for cfg in L.CONFIGS.values():
        names = {s.name: tuple(s.shape) for s in build_model(config_from_dict(cfg)).tensor_specs()}
        made = L.random_weights(cfg, 1)
        assert {n: tuple(t.shape) for n, t in made.items()} == names


def test_missing_and_unexpected_tensors_are_one_report(tmp_path):
    from lgml_b200.weights import WeightError
    from lgml_b200.weights.loader import check_index
    from lgml_b200.weights.safetensors import index_folder

    weights = L.random_weights(L.ALL_DELTA, 3)
    weights.pop("l1.mix.A_log")
    weights["l1.mlp.router"] = torch.zeros(2, 96)       # that layer has no feed-forward
    weights["l0.hc1.mix"] = torch.zeros(3, 3)
    folder = L.write_folder(tmp_path / "m", L.ALL_DELTA, weights)
    with pytest.raises(WeightError) as e:
        check_index(index_folder(folder), build_model(config_from_dict(L.ALL_DELTA)).tensor_specs())
    assert e.value.missing == ["l1.mix.A_log"] and e.value.unexpected == ["l1.mlp.router"] and [w[0] for w in e.value.wrong_shape] == ["l0.hc1.mix"]


@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 64), (8.0, 0.5, 2.0, 300), (2.0, 1.0, 32.0, 4096)])
def test_blended_frequencies(scaling):
    rot = {"base": 700.0, "dims": 24}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    part = rotation_of(32, rot)
    ff = frequency_factors(32, 700.0, part.scaling, 24)
    mine = [700.0 ** (-2.0 * i / 24) / f for i, f in enumerate(ff)]
    assert np.allclose(mine, P.banded_frequencies(700.0, 24, rot.get("scaling")), rtol=1e-12)
    if scaling and scaling[3] in (64, 300):
        assert len(set(np.round(ff, 6))) > 2, "this case should reach all three bands"


def test_a_pair_of_mixers_keeps_pages_on_one_side_only():
    side = lambda: make_part("mixer", "normed_attention", width=16, n_heads=2, n_kv_heads=1, head_dim=8, v_head_dim=8, scale=1.0,
                             position=make_part("position", "rope", head_dim=8, theta=100.0), eps=1e-5)
    with pytest.raises(TypeError):
        make_part("mixer", "summed", width=16, left=side(), right=side())
    with pytest.raises(ValueError):
        make_part("feed_forward", "routed_experts", width=16, inner=8, n_experts=2, top=5, n_identity=2)
    with pytest.raises(ValueError):
        make_part("block", "hyper", streams=9, mixer_norm=None, mixer=None)


def test_plain_functions_against_closed_forms():
    x = np.array([[1.0, 2.0, 3.0, 6.0]])
    assert np.allclose(P.norm_one_plus(x, np.full(4, 0.5), 0.0), 1.5 * x / math.sqrt(12.5))
    # streams: mix is indexed [from, to]
    X = np.array([[[1.0], [10.0]]])
    mix = np.array([[1.0, 2.0], [3.0, 4.0]])
    new = P.streams_write(X, np.array([[100.0]]), np.array([1.0, 0.5]), mix)
    assert np.allclose(new[0, :, 0], [1 + 30 + 100, 2 + 40 + 50])
    assert np.allclose(P.streams_read(X, np.array([2.0, -1.0])), [[-8.0]])
    # a mask of size 3 that keeps two first tokens
    seen = [[bool(P.visible(i, j, 3, 2)) for j in range(7)] for i in range(7)]
    assert seen[6] == [True, True, False, False, True, True, True] and seen[1] == [True, True] + [False] * 5
    assert all(bool(P.visible(50, j, 0, 0)) for j in range(51))
    # one key, a sink of equal weight: half the value comes through
    one = np.ones((1, 1, 2))
    assert np.allclose(P.sink_window_attention(one, one, np.full((1, 1, 3), 4.0), 1.0, [2.0], 5, 0), 2.0)
    # delta rule: writing the same unit key twice with beta 1 replaces its value
    k = np.array([[[1.0, 0.0]], [[1.0, 0.0]]])
    o = P.delta_scan(k, k, np.array([[[5.0]], [[-3.0]]]), np.ones((2, 1)), np.ones((2, 1)))
    assert np.allclose(o[:, 0, 0], [5.0, -3.0])
    # matrix memory: one token with an input gate far below zero.  m starts at 0, so m = max(f, i) = f here, and exp(-m) decides
    q = k1 = np.ones((1, 1, 1))
    o = P.matrix_memory_scan(q, k1, np.full((1, 1, 1), 2.0), np.full((1, 1), -9.0), np.full((1, 1), -0.5))
    b = math.exp(-9.0 + 0.5)
    assert np.allclose(o, 2.0 * b / (math.exp(0.5) + 1e-6))
    # and with a large one: n . q outweighs it
    o = P.matrix_memory_scan(q * 3, k1, np.full((1, 1, 1), 2.0), np.full((1, 1), 4.0), np.full((1, 1), -0.5))
    assert np.allclose(o, 6.0 / (3.0 + 1e-6))
    # router: the correction moves the choice, not the weight; the weights are not renormalised
    W = {"p.router": np.array([[2.0], [1.0], [0.0]]), "p.correction": np.array([0.0, -1.0, 0.0])}
    ids, w = P.route(np.ones((1, 1)), W, "p", 2)
    s = np.exp([2.0, 1.0, 0.0]) / np.exp([2.0, 1.0, 0.0]).sum()
    assert ids.tolist() == [[0, 2]] and np.allclose(w, s[[0, 2]])
    W.update({"p.e0.gate": np.ones((1, 1)), "p.e0.up": np.ones((1, 1)), "p.e0.down": np.ones((1, 1))})
    y = P.experts(np.full((1, 1), 1.0), W, "p", {"router": {"experts": 1, "identity": 2, "top": 2}})
    assert np.allclose(y, s[0] * P.silu(1.0) + s[2])
