"""Zudovik without a GPU: its configuration, what its layers ask of the cache, the tensors it declares, errors that name the
key, and the plain implementation's own mechanisms against cases worked by hand."""
import copy
import math

import numpy as np
import pytest

from friday_inference_engine_b200 import ConfigError, describe_model, read_config

import plain_zudovik as plain
import zudovik_models as zm

CFG = zm.CONFIGS["P"]


def test_the_name_selects_the_design():
    assert read_config(CFG)["architecture"] == "Zudovik"
    d = describe_model(CFG)
    assert d["architecture"] == "Zudovik" and d["n_layers"] == 5
    # layers 3 and 4 read the entries that layers 2 and 0 fill
    assert [(c["layer"], c["cache"], c["write"]) for c in d["program"]] == [(0, 0, True), (1, 1, True), (2, 2, True), (3, 2, False), (4, 0, False)]


def test_cache_requests():
    reqs = describe_model(CFG)["cache_requests"]
    assert set(reqs) == {"0", "1", "2"}                       # nothing is kept for the layers that read another's keys
    assert reqs["0"] == {"kind": "kv", "n_kv_heads": 2, "head_dim": 16, "window": 0, "v_head_dim": 24, "keep_first": 0}
    assert reqs["1"] == {"kind": "state", "shape": [3 * 16 * 24], "dtype": "float32"}
    assert reqs["2"] == {"kind": "kv", "n_kv_heads": 3, "head_dim": 20, "window": 0, "v_head_dim": 12, "keep_first": 0}


def test_declared_tensors():
    """Exactly the tensors that the tests' writer makes, with their shapes."""
    for name, cfg in zm.CONFIGS.items():
        shapes = {p["name"]: p["shape"] for p in describe_model(cfg)["params"]}
        made = {n: list(x.shape) for n, x in zm.tensors_of(cfg, np.random.default_rng(0)).items()}
        assert shapes == made, name
    d = describe_model(CFG)
    shapes = {p["name"]: p["shape"] for p in d["params"]}
    assert shapes["l0.mix.q.norm"] == [64] and shapes["l0.mix.k.norm"] == [32] and shapes["l0.mix.g"] == [4, 96] and shapes["l0.mix.sink"] == [4]
    assert "l3.mix.k" not in shapes and "l3.mix.v.b" not in shapes and "l3.mix.k.norm" not in shapes and shapes["l3.mix.q.norm"] == [120]
    assert shapes["l1.mlp.router"] == [8, 96] and shapes["l1.mlp.correction"] == [8] and "l1.mlp.e6.gate" not in shapes
    assert shapes["l1.mlp.shared.sg"] == [1, 96] and "l3.mlp.shared.sg" not in shapes
    assert "l2.norm2" in d["ignorable"] and "l2.norm2" not in shapes


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c["layers"][0].update(type="retention"), "retention"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "share"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=1.0), "base"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5]), "decay"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "shape"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "gated"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "choices"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
])
def test_bad_config_names_the_key(change, word):
    cfg = copy.deepcopy(CFG)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        read_config(cfg)
    assert word in str(e.value)


# ---- the plain implementation's mechanisms against cases worked by hand
def test_plain_states_decay_and_add():
    k = np.array([[1.0, 0.0], [0.0, 2.0], [1.0, 1.0]])
    v = np.array([[3.0], [5.0], [7.0]])
    S = plain.decayed_states(k, v, 0.5)
    assert np.allclose(S[0], [[3.0], [0.0]]) and np.allclose(S[1], [[1.5], [10.0]]) and np.allclose(S[2], [[7.75], [12.0]])
    assert np.allclose(plain.decayed_states(k, v, 0.0)[2], [[7.0], [7.0]])


def test_plain_rotation_pairs_neighbours():
    x = np.zeros((2, 1, 6))
    x[1, 0] = [1.0, 0.0, 0.0, 1.0, 5.0, 6.0]
    y = plain.rotate_neighbours(x, {"base": 100.0, "dims": 4})
    a, b = 1.0, 100.0 ** -0.5
    assert np.allclose(y[1, 0], [math.cos(a), math.sin(a), -math.sin(b), math.cos(b), 5.0, 6.0]) and np.allclose(y[0], 0.0)


def test_plain_cap_and_sink():
    assert np.allclose(plain.cap(np.array([0.0, 1e-4, 1e6, -1e6]), 4.0), [0.0, 1e-4, 4.0, -4.0])
    p = plain.softmax_with_sink(np.array([[1.0, 9.0], [1.0, 2.0]]), 3.0)
    z = math.exp(1.0) + math.exp(2.0) + math.exp(3.0)
    assert np.allclose(p[1], [math.exp(1.0) / z, math.exp(2.0) / z])
    assert np.allclose(p[0], [math.exp(1.0) / (math.exp(1.0) + math.exp(3.0)), 0.0])        # causal; the sink counts once


def test_plain_choice():
    z = np.log(np.array([0.4, 0.3, 0.2, 0.1]))
    ids, w = plain.choose(z, np.array([0.0, 0.0, 0.0, 0.25]), 2)
    assert list(ids) == [0, 3] and np.allclose(w, [0.8, 0.2])          # chosen with the correction, weighted without it


def test_plain_clipped_unit_and_identity_expert():
    W = {"gate": np.array([[2.0]]), "up": np.array([[-3.0]]), "down": np.array([[1.0]])}
    g, u = 0.5, -0.5                                                    # min(2, 0.5), clamp(-3, +-0.5)
    assert np.isclose(plain.clipped_glu(np.array([1.0]), W, 0.5)[0], g / (1.0 + math.exp(-1.702 * g)) * (u + 1.0))
    assert np.isclose(plain.clipped_glu(np.array([-1.0]), W, 0.5)[0], -2.0 / (1.0 + math.exp(1.702 * 2.0)) * 1.5)      # the gate has no lower limit
    mlp = {"router": {"experts": 1, "identity": 1, "top": 1}, "expert": {"limit": 1.0}}
    h = np.array([[4.0]])
    full = dict({"e0." + n: x for n, x in W.items()}, router=np.array([[0.0], [1.0]]), correction=np.zeros(2))
    assert np.allclose(plain.experts(h, full, mlp), h)                 # the identity expert alone, weight one


def test_plain_whole_norm_spans_the_heads():
    x = np.array([[3.0, 4.0, 0.0, 0.0]])
    assert np.allclose(plain.rms(x, np.ones(4), 0.0), x / 2.5)
