"""Dapozen without a GPU: its configuration, what its layers ask of the cache, the tensors it declares, errors that name the
key, the cache's books for runs of positions, and the plain implementation's own mechanisms against cases worked by hand."""
import copy
import math

import numpy as np
import pytest

from friday_inference_engine_b200 import ConfigError, describe_model, read_config
from friday_inference_engine_b200.cache import CacheBook, kv_request

import dapozen_models as dm
import plain_dapozen as plain
import tiny_configs

CFG = dm.CONFIGS["P"]


def test_the_name_selects_the_design():
    assert read_config(CFG)["architecture"] == "Dapozen"
    d = describe_model(CFG)
    assert d["architecture"] == "Dapozen" and d["n_layers"] == 4
    # layers 1 and 2 run twice, every run with an entry of its own
    assert [(c["layer"], c["cache"], c["write"]) for c in d["program"]] == [(0, 0, True), (1, 1, True), (2, 2, True), (1, 3, True), (2, 4, True), (3, 5, True)]
    assert [c["layer"] for c in d["program"]] == plain.run_order(CFG)
    assert [c["layer"] for c in describe_model(dm.CONFIGS["Q"])["program"]] == [0, 1, 2]


def test_cache_requests():
    reqs = describe_model(CFG)["cache_requests"]
    assert set(reqs) == {"0", "1", "2", "3", "4", "5"}
    assert reqs["0"] == {"kind": "several", "parts": [
        {"kind": "kv", "n_kv_heads": 2, "head_dim": 16, "window": 0, "v_head_dim": 24, "keep_first": 0, "chunk": 10},
        {"kind": "state", "shape": [3 * (6 * 16 + 2 * 24)], "dtype": "float32"}]}
    # the convolution's two inputs of x, B and C, then the heads' matrices
    assert reqs["1"] == {"kind": "state", "shape": [2 * (48 + 2 * 32) + 6 * 16 * 8], "dtype": "float32"} and reqs["3"] == reqs["1"]
    assert reqs["2"]["parts"][0]["chunk"] == 37 and reqs["2"]["parts"][1]["shape"] == [9 * 20 + 3 * 12]
    one_tap = describe_model(dm.CONFIGS["Q"])["cache_requests"]
    assert one_tap["0"]["shape"] == [32 * 8] and one_tap["1"]["parts"][0]["chunk"] == 1


def test_declared_tensors():
    """Exactly the tensors that the tests' writer makes, with their shapes."""
    for name, cfg in dm.CONFIGS.items():
        shapes = {p["name"]: p["shape"] for p in describe_model(cfg)["params"]}
        made = {n: list(x.shape) for n, x in dm.tensors_of(cfg, np.random.default_rng(0)).items()}
        assert shapes == made, name
    d = describe_model(CFG)
    shapes = {p["name"]: p["shape"] for p in d["params"]}
    assert shapes["l0.mix.q.conv"] == [64, 4] and shapes["l0.mix.v"] == [48, 96] and shapes["l0.mix.g"] == [96, 96] and "l0.mix.g.b" not in shapes
    assert shapes["l1.mix.in"] == [2 * 48 + 2 * 32 + 6, 96] and shapes["l1.mix.conv"] == [112, 3] and shapes["l1.mix.norm"] == [48]
    assert shapes["l1.mlp.table"] == [300, 3] and shapes["l1.mlp.shared.up"] == [40, 96] and "l1.mlp.router" not in shapes
    assert "l2.norm2" in d["ignorable"] and "l2.norm2b" in d["ignorable"] and "l2.norm2" not in shapes


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["layers"][0].update(type="retention"), "retention"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "share"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=1.0), "base"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "equal parts"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "gated"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "choices"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
])
def test_bad_config_names_the_key(change, word):
    cfg = copy.deepcopy(CFG)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        read_config(cfg)
    assert word in str(e.value)


def test_random_folders_hold_a_table_of_different_experts(tmp_path):
    cfg = dict(CFG)
    tiny_configs.make_model_dir(str(tmp_path), cfg, 4)
    _, t = plain.load(str(tmp_path))
    table = t["l1.mlp.table"]
    assert table.shape == (300, 3) and table.min() == 0 and table.max() == 5
    assert all(len(set(row)) == 3 for row in table)
    assert len({tuple(row) for row in table}) > 3


def test_the_cache_gives_pages_back_at_the_end_of_a_run():
    """Runs of 150 positions: a page goes back as soon as the sequence's next position begins a run behind it."""
    book = CacheBook({0: kv_request(2, 16, chunk=150), 1: kv_request(2, 16)}, max_tokens=2048, max_seq_tokens=1024, max_slots=2)
    s = book.alloc_slot()

    def pages(g):
        return [lp for lp, page in enumerate(book.info()["groups"][g]["table"][s]) if page >= 0]

    def go(n):
        book.reserve([s], [n])
        book.commit([s], [n])

    go(149)
    assert pages(0) == [0, 1, 2] and pages(1) == [0, 1, 2]
    go(1)                                          # 150 tokens: the next position begins the second run, in page 2
    assert pages(0) == [2] and pages(1) == [0, 1, 2]
    go(149)
    assert pages(0) == [2, 3, 4]
    go(1)                                          # 300 tokens: the third run begins in page 4
    assert pages(0) == [4]
    go(400)                                        # across whole runs: 700 tokens, the run from 600 on (page 9)
    assert pages(0) == [9, 10] and pages(1) == list(range(11))
    book.free_slot(s)
    info = book.info()
    assert all(g["pages_held"] == 0 for g in info["groups"])


def test_a_run_and_a_window_do_not_go_together():
    with pytest.raises(Exception) as e:
        CacheBook({0: kv_request(2, 16, window=8, chunk=16)}, max_tokens=256, max_seq_tokens=256)
    assert "runs of positions" in str(e.value)


# ---- the plain implementation's mechanisms against cases worked by hand
def test_plain_convolution():
    u = np.array([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]])
    y = plain.causal_conv(u, np.array([[0.5, 2.0], [1.0, 0.0]]))       # the last tap is the present row's
    assert np.allclose(y, [[2.0, 0.0], [4.5, 10.0], [7.0, 20.0]])


def test_plain_runs_of_positions():
    p = plain.chunk_softmax(np.log(np.array([[1.0, 9, 9, 9], [1, 3, 9, 9], [9, 9, 1, 9], [9, 9, 1, 1]])), 2)
    assert np.allclose(p, [[1, 0, 0, 0], [0.25, 0.75, 0, 0], [0, 0, 1, 0], [0, 0, 0.5, 0.5]])


def test_plain_rotation_pairs_neighbours():
    x = np.zeros((2, 1, 6))
    x[1, 0] = [1.0, 0.0, 0.0, 1.0, 5.0, 6.0]
    y = plain.rotate_neighbours(x, {"base": 100.0, "dims": 4})
    a, b = 1.0, 100.0 ** -0.5
    assert np.allclose(y[1, 0], [math.cos(a), math.sin(a), -math.sin(b), math.cos(b), 5.0, 6.0]) and np.allclose(y[0], 0.0)


def test_plain_states():
    x, B = np.array([[3.0], [5.0]]), np.array([[1.0, 0.0], [0.0, 2.0]])
    S = plain.ssd_states(x, B, np.array([1.0, 0.5]), math.log(math.log(4.0)))       # decays 1/4 and 1/2
    assert np.allclose(S[0], [[3.0], [0.0]]) and np.allclose(S[1], [[1.5], [5.0]])
    assert np.isclose(plain.softplus(0.0), math.log(2.0)) and np.isclose(plain.softplus(50.0), 50.0)


def test_plain_norm_in_parts():
    y = plain.group_norm(np.array([[3.0, 4.0, 0.0, 2.0]]), 2, np.array([1.0, 1.0, 1.0, 10.0]), 0.0)
    assert np.allclose(y, [[3.0 / math.sqrt(12.5), 4.0 / math.sqrt(12.5), 0.0, 10.0 * math.sqrt(2.0)]])


def test_plain_experts_by_table():
    unit = {"gate": np.array([[2.0]]), "up": np.array([[-3.0]]), "down": np.array([[1.0]])}
    g, u = 0.5, -0.5                                                    # min(2, 0.5), clamp(-3, +-0.5)
    one = g / (1.0 + math.exp(-1.702 * g)) * (u + 1.0)
    assert np.isclose(plain.clipped_glu(np.array([1.0]), unit, 0.5)[0], one)
    assert np.isclose(plain.clipped_glu(np.array([-1.0]), unit, 0.5)[0], -2.0 / (1.0 + math.exp(1.702 * 2.0)) * 1.5)      # the gate has no lower limit
    W = {"e%d.%s" % (e, n): x * (e + 1 if n == "down" else 1) for e in range(3) for n, x in unit.items()}
    W["table"] = np.array([[0, 2], [1, 0]])
    mlp = {"router": {"experts": 3, "top": 2}, "expert": {"limit": 0.5}}
    y = plain.experts(np.array([[1.0], [1.0]]), [1, 0], W, mlp)
    assert np.allclose(y, [[one * 1.5], [one * 2.0]])                   # (2 + 1) / 2 and (1 + 3) / 2


def test_plain_logits_are_capped():
    cfg = dm.CONFIGS["dense_only"]
    t = dm.tensors_of(cfg, np.random.default_rng(1))
    raw = plain.forward(dict(cfg, logit_softcap=None), t, [3, 4])
    assert np.allclose(plain.forward(cfg, t, [3, 4]), 12.0 * np.tanh(raw / 12.0))
