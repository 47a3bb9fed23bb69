"""Nelosun on the host: the registry, the configuration's keys and errors, the order in which looped layers run and which cache and
state each run gets, the tensors the model asks for, random-weights folders with integer tables, and the plain functions
against closed forms."""
import copy
import math

import numpy as np
import pytest
import torch

from lgml_b200.cache import FixedState, PagedKV
from lgml_b200.config import ConfigError, NelosunConfig, architectures, config_from_dict, load_config
from lgml_b200.models import LayerCall, DecoderModel, build_model
from lgml_b200.parts import TableRouting
from lgml_b200.weights import INT_TABLE, TensorSpec, WeightError, index_folder, load_tensors, random_tensors, read_tensor, write_random_model
from lgml_b200.weights.loader import check_index
from tests import nelosun_helpers as L
from tests.plain import nelosun_plain as P


def test_registered_and_read_from_its_own_keys():
    assert "Nelosun" in architectures()
    cfg = config_from_dict(copy.deepcopy(L.LOOPED))
    assert isinstance(cfg, NelosunConfig)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.num_hidden_layers, cfg.embed_scale, cfg.norm_eps, cfg.loop) == (97, 64, 4, 3.0, 1e-5, (1, 3, 3))
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    plain = config_from_dict(copy.deepcopy(L.ODD))
    assert (plain.embed_scale, plain.loop) == (1.0, None)


@pytest.mark.parametrize("edit,word", [
    (lambda d: d.pop("width"), "width"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d.update(embedding=3.0), "embedding"),
    (lambda d: d["embedding"].update(scale="x"), "scale"),
    (lambda d: d["layers"][0].update(type="conv"), "layers[0].type"),
    (lambda d: d["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda d: d["layers"][0]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda d: d["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["rot"].pop("base"), "base"),
    (lambda d: d["layers"][2]["mixer"].update(blocks=5), "blocks"),
    (lambda d: d["layers"][2]["mixer"].pop("conv"), "conv"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda d: d["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda d: d["layers"][0]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda d: d["loop"].update(stop=6), "loop"),
    (lambda d: d["loop"].update(start=3), "loop"),
    (lambda d: d["loop"].update(times=0), "loop"),
    (lambda d: d["loop"].pop("times"), "loop.times"),
])
def test_errors_name_the_key(edit, word):
    d = copy.deepcopy(L.LOOPED)
    edit(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert word in str(e.value)


def test_looped_layers_run_in_order_and_every_run_has_its_own_cache_and_state():
    cfg = config_from_dict(copy.deepcopy(L.LOOPED))
    runs = cfg.layer_runs()
    assert [i for i, _ in runs] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [n for _, n in runs] == [None, 0, None, 1, None, 2, None, None]
    assert [(i, n is not None) for i, n in runs] == P.layer_runs(L.LOOPED)
    model = build_model(cfg)
    assert [(c.block, c.begins_pass, c.cache) for c in model.schedule] == [(i, n, None) for i, n in runs]
    layout = model.cache_layout()
    assert sorted(layout) == list(range(8))                            # one entry per run, not per layer
    assert layout[0] == PagedKV(2, 16, None, 24) and layout[7] == PagedKV(2, 24, None, 8)
    for run in (1, 3, 5):
        assert layout[run] == PagedKV(1, 24 + 8, None, 24, v_in_k=True)
    for run in (2, 4, 6):
        assert layout[run] == FixedState((48 + 4 * 48,), torch.float32)       # the recurrence, then the ring of the four taps
    # a loop from the first layer on, one that runs once, and none
    assert [n for _, n in config_from_dict(copy.deepcopy(L.ALL_LOOP)).layer_runs()] == [0, None, None, 1, None, None]
    assert [n for _, n in config_from_dict(copy.deepcopy(L.WIDE_HEADS)).layer_runs()] == [None, None, 0, None, None]
    free = build_model(config_from_dict(copy.deepcopy(L.ODD)))
    assert free.pass_input is None and free.cache_layout()[3] == FixedState((37,), torch.float32)       # one tap keeps no inputs


def test_a_pass_needs_the_part_that_begins_it():
    model = build_model(config_from_dict(copy.deepcopy(L.ODD)))
    with pytest.raises(ValueError):
        DecoderModel(model.config, model.embedding, model.blocks, model.final_norm, model.head, schedule=[LayerCall(0, begins_pass=0)])


def test_which_parts_a_configuration_asks_for():
    model = build_model(config_from_dict(copy.deepcopy(L.LOOPED)))
    a, lat, rec, b = model.blocks
    m = a.mixer
    assert (m.n_heads, m.n_kv_heads, m.head_dim, m.v_head_dim, m.scale, m.temp_coef, m.temp_every, m.gate_cols) == (6, 2, 16, 24, 0.3, 0.7, 13, 6)
    assert m.sink_score == 0.0 and not m.has_sink and m.out_bias and m.slope_base is None and b.mixer.temp_coef == 0.0
    assert (lat.mixer.q_rank, lat.mixer.rank, lat.mixer.halves, lat.mixer.rope_dims, lat.mixer.scale) == (20, 24, True, 8, 0.25) and lat.ffn is None
    assert (rec.mixer.inner, rec.mixer.blocks, rec.mixer.taps) == (48, 3, 4)
    assert (a.ffn.n_experts, a.ffn.top, a.ffn.inner, a.ffn.clamp) == (5, 2, 24, (1.702, 0.9)) and a.ffn.routing is rec.ffn.routing
    assert model.head.tied_to is model.embedding and model.embed_scale == 3.0


def test_folder_of_random_weights_and_the_loaders_report(tmp_path):
    cfg = config_from_dict(copy.deepcopy(L.ODD))
    folder = write_random_model(tmp_path / "m", cfg, seed=3)
    loaded = load_config(folder)
    assert loaded.to_dict() == cfg.to_dict()
    specs = build_model(loaded).tensor_specs()
    index = index_folder(folder)
    check_index(index, specs)
    names = set(index)
    assert {"embed", "final.norm", "l0.norm1", "l0.ls1", "l0.ls2", "l0.mix.lam", "l0.mix.ra.b", "l0.mix.conv.b", "l1.mix.o.b", "l1.mix.g", "l1.mlp.table",
            "l1.mlp.e5.down", "l2.mix.dq.norm", "l2.mix.uq", "l3.ls1"} <= names
    assert not {"head", "loop.in", "l3.ls2", "l3.mlp.table", "l1.mix.sink", "l1.mix.vmix", "l2.mix.q", "l0.norm2"} & names
    assert tuple(index["l1.mix.g"].shape) == (3, 37) and tuple(index["l0.mix.ri"].shape) == (3, 7, 7) and tuple(index["l1.mlp.table"].shape) == (61, 3)
    table = read_tensor(index["l1.mlp.table"])
    assert table.dtype == torch.int32 and int(table.min()) >= 0 and int(table.max()) < 6
    assert all(len(set(row.tolist())) == 3 for row in table) and len(set(map(tuple, table.tolist()))) > 20
    tensors = load_tensors(folder, specs, torch.bfloat16, "cpu")
    assert tensors["l1.mlp.table"].dtype == torch.int32 and tensors["l0.mix.ra"].dtype == torch.bfloat16 and tensors["l0.mix.lam"].dtype == torch.float32
    # the vector of an absent feed-forward may lie in the folder unread
    spec = {s.name: s for s in specs}
    assert spec["l3.ls2"].optional and not spec["l0.ls2"].optional
    index.pop("l2.mlp.table")
    index["l9.extra"] = index["embed"]
    with pytest.raises(WeightError) as e:
        check_index(index, specs)
    assert e.value.missing == ["l2.mlp.table"] and e.value.unexpected == ["l9.extra"]


def test_integer_tables_of_the_random_weights_mode():
    spec = TensorSpec("t", (50, 4), INT_TABLE, below=4)
    a, b = (random_tensors([spec], seed)["t"] for seed in (1, 1))
    assert torch.equal(a, b) and all(sorted(row.tolist()) == [0, 1, 2, 3] for row in a)
    assert not torch.equal(a, random_tensors([spec], 2)["t"])
    with pytest.raises(ValueError):
        random_tensors([TensorSpec("t", (50, 4), INT_TABLE, below=3)], 1)


def test_tables_that_name_no_expert_are_refused():
    routing = TableRouting()
    assert routing.add(torch.tensor([[0, 2], [1, 0]], dtype=torch.int32), 3) == 0
    for bad, n in (([[0, 3], [1, 0]], 3), ([[0, -1], [1, 0]], 3)):
        with pytest.raises(ValueError):
            routing.add(torch.tensor(bad, dtype=torch.int32), n)
    with pytest.raises(ValueError):
        routing.add(torch.zeros((3, 1), dtype=torch.int32), 1)             # another vocabulary


def test_plain_functions_against_closed_forms():
    # one is added to the denominator: a single key of score 0 gets half, of score ln 3 three quarters, very negative ones nothing
    see = np.ones((1, 2), dtype=bool)
    w = P.softmax_plus_one(np.array([[0.0, -np.inf]]), see)
    assert np.allclose(w, [[0.5, 0.0]])
    assert np.allclose(P.softmax_plus_one(np.array([[math.log(3.0), -900.0]]), see), [[0.75, 0.0]])
    assert np.allclose(P.softmax_plus_one(np.array([[-800.0, -801.0]]), see), 0.0) and np.allclose(P.softmax_plus_one(np.array([[900.0, 900.0]]), see), 0.5)
    # the temperature steps where (p + 1) / every passes a whole number
    t = P.query_temperature(9, 2.0, 4)
    assert np.allclose(t, 1.0 + 2.0 * np.log([1, 1, 1, 2, 2, 2, 2, 3, 3]))
    # rotation: entry i turns with entry i + dims / 2
    v = np.zeros((3, 5)); v[:, 0] = 1.0; v[:, 1] = 1.0; v[:, 4] = 7.0
    r = P.rotate_half(v, 100.0, 4, [0, 1, 2])
    assert np.allclose(r[2], [np.cos(2.0), np.cos(0.2), np.sin(2.0), np.sin(0.2), 7.0])
    # the convolution: the last column weighs the current token
    u = P.causal_conv(np.array([[1.0], [10.0], [100.0]]), np.array([[2.0, 3.0]]), np.array([0.5]))
    assert np.allclose(u[:, 0], [3.5, 32.5, 320.5])
    # the recurrence: r = 1, softplus(lam) = ln 2 / 8 -> a = 1/2, the pushed part sqrt(3)/2 i u
    lam = np.log(np.expm1(np.log(2.0) / 8.0))
    S = P.rglru_scan(np.array([[2.0], [4.0]]), np.ones((2, 1)), np.array([[1.0], [0.5]]), np.array([lam]))
    k = math.sqrt(0.75)
    assert np.allclose(S[:, 0], [2.0 * k, 0.5 * 2.0 * k + 2.0 * k])
    # a square matrix per part
    w = np.zeros((2, 2, 2)); w[0, 0, 1] = 1.0; w[1] = np.eye(2) * 3.0
    assert np.allclose(P.block_linear(np.array([[1.0, 2.0, 3.0, 4.0]]), w, np.array([[0.1, 0.2], [0.3, 0.4]])), [[2.1, 0.2, 9.3, 12.4]])
    # an expert: the gate is cut from above only, the up branch on both sides
    W = {"e.gate": np.array([[1.0]]), "e.up": np.array([[1.0]]), "e.down": np.array([[1.0]])}
    act = lambda g, u: g / (1.0 + math.exp(-1.702 * g)) * (u + 1.0)
    assert np.allclose(P.clamped_expert(np.array([[5.0], [-5.0], [0.5]]), W, "e", 2.0), [[act(2.0, 2.0)], [act(-5.0, -2.0)], [act(0.5, 0.5)]])
    # the table: each of a token's experts counts 1 / top
    W = {"f.table": np.array([[1, 0], [2, 1]])}
    for e in range(3):
        W[f"f.e{e}.gate"], W[f"f.e{e}.up"], W[f"f.e{e}.down"] = np.array([[1.0]]), np.array([[0.0]]), np.array([[10.0 ** e]])
    y = P.table_experts(np.array([[1.0], [1.0]]), [1, 0], W, "f", {"router": {"top": 2}, "expert": {"limit": 9.0}})
    assert np.allclose(y, act(1.0, 0.0) * np.array([[55.0], [5.5]]))
    # passes: layers 1 and 2 twice, x made anew before layer 1 each time
    assert P.layer_runs({"layers": [0, 0, 0, 0], "loop": {"start": 1, "stop": 3, "times": 2}}) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
