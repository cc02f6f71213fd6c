"""Rurunex without a GPU: configuration, weight packing, registry, and the oracle's own consistency."""
import json
import math

import numpy as np
import pytest

from oracle import rurunex_ref as R


def small_config(**kw):
    rot = {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0, "original": 16, "fast": 4.0, "slow": 1.0}}
    att = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "mask": {"size": 5}, "rot": rot, "scale": 0.4, "softcap": 3.0}
    cfg = {"architecture": "Rurunex", "embedding": {"scale": 2.5}, "vocab": 19, "width": 22, "norm": {"eps": 1e-5}, "logit_scale": 0.25,
           "layers": [{"type": "attention", "mixer": att, "mlp": {"kind": "dense", "ff": 9}},
                      {"type": "gla", "mixer": {"heads": 2, "dim": 5, "vdim": 4, "tau": 3.0}, "mlp": None},
                      {"type": "channel_delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "conv": 3}, "mlp": {"kind": "dense", "ff": 7}},
                      {"type": "attention", "mixer": {**att, "kv_from": 0, "mask": {"size": 9}}, "mlp": None}]}
    cfg.update(kw)
    return cfg


def test_registry_and_shape_errors(gpu, tmp_path):
    from applegpu_runtime_b200 import models
    cfg = small_config()
    assert models.architecture_of(cfg) == "Rurunex"
    w = gpu.init_rurunex_weights(cfg)
    assert "l3.mix.k" not in w and "l3.mix.q.norm" in w and "l1.norm2" not in w
    for name in ("l0.mix.k.norm", "l2.mix.v.conv", "l1.mix.a1", "l0.norm2b", "l2.mlp.up", "l2.mix.g1"):
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            gpu.load_rurunex(cfg, {k: v for k, v in w.items() if k != name})
    with pytest.raises(ValueError, match="shape"):
        gpu.load_rurunex(cfg, {**w, "l2.mix.dt_bias": np.zeros(4, np.float32)})
    for change, text in ((("type", "other"), "unknown mixer"), (("mixer", {**cfg["layers"][0]["mixer"], "kv_heads": 3}), "heads over"),
                         (("mixer", {**cfg["layers"][0]["mixer"], "rot": {"dims": 8, "base": 10.0}}), "rotated dimensions")):
        bad = json.loads(json.dumps(cfg))
        bad["layers"][0][change[0]] = change[1]
        with pytest.raises(ValueError, match=text):
            gpu.load_rurunex(bad, w)


def test_layer_records():
    from applegpu_runtime_b200.seqmodel import LAYER_WEIGHTS, ROTATION, Layer, Tensors
    layer = Layer("key_decay", 1, 1, 1, norm1="n1", post2="p2", w_down="d", own=["a", "b", "c", "e"])
    r = layer.weights()
    assert len(r) == LAYER_WEIGHTS and r[0] == "n1" and r[5:8] == ["a", "b", "c"] and r[9:12] == ["p2", "d", "e"] and r[ROTATION] == "c"
    t = Tensors({"x": np.zeros((3, 2), np.float32)})
    assert t.rank("x") == 3
    with pytest.raises(ValueError):
        t.rank("y")


def test_oracle_portions_agree(gpu):
    cfg = small_config()
    w = gpu.init_rurunex_weights(cfg, seed=1, std=0.4, ranks={"gla": 3, "channel_delta": 2})
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 24)
    want = R.forward(cfg, w, toks)
    states, got = [], []
    for lo, hi in ((0, 5), (5, 6), (6, 8), (8, 24)):
        got.append(R.forward(cfg, w, toks[lo:hi], states))
    assert np.max(np.abs(np.concatenate(got) - want)) < 1e-10


def test_oracle_delta_rule_replaces_what_a_key_returns():
    """Writing twice under the same unit key with full strength leaves the second value only; decays act ahead of the write."""
    k = np.array([[[0.6, 0.8]], [[0.6, 0.8]]])
    v = np.array([[[3.0, -1.0]], [[5.0, 2.0]]])
    one = np.ones((2, 1, 2))
    o, S = R.delta_recurrence(k, k, v, one, np.ones((2, 1)), np.zeros((1, 2, 2)))
    assert np.allclose(o[1, 0], v[1, 0]) and np.allclose(S[0].T @ k[1, 0], v[1, 0])
    o, _ = R.gla_recurrence(k, k, v, np.full((2, 1, 2), 0.5), np.zeros((1, 2, 2)))
    assert np.allclose(o[1, 0], 0.5 * v[0, 0] + v[1, 0])


def test_oracle_window_cap_and_halves():
    rng = np.random.default_rng(2)
    q, k, v = rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 1, 4)), rng.standard_normal((6, 1, 3))
    full = R.attention_rows(q, k, v, 0, 0.5, 2.0, None)
    assert np.allclose(R.attention_rows(q, k, v, 0, 0.5, 2.0, 6), full)
    assert np.allclose(R.attention_rows(q, k, v, 0, 0.5, 2.0, 1), np.repeat(v, 2, axis=1))
    assert np.allclose(R.attention_rows(q[5:], k[3:], v[3:], 2, 0.5, 2.0, 3)[0], R.attention_rows(q, k, v, 0, 0.5, 2.0, 3)[5])
    x = np.zeros((1, 1, 4))
    x[0, 0, 0] = 1.0
    y = R.rotate_halves(x, [3], {"dims": 4, "base": 10.0})[0, 0]
    assert math.isclose(y[0], math.cos(3)) and math.isclose(y[2], math.sin(3)) and y[1] == y[3] == 0.0
