"""Gedenex without a GPU: configuration, weight packing, rotation tables, file format, registry, and the oracle's own consistency."""
import json
import math

import numpy as np
import pytest

from oracle import gedenex_ref as R


def small_config(**kw):
    cfg = {"architecture": "Gedenex", "vocab": 19, "width": 22, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 2, "times": 2},
           "layers": [{"type": "latent_attention", "mlp": None,
                       "mixer": {"heads": 2, "dim": 5, "rot_dim": 4, "vdim": 3, "kv_rank": 7, "scale": 0.4, "rot": {"dims": 4, "base": 100.0}}},
                      {"type": "mlstm", "mlp": {"kind": "dense", "ff": 9, "limit": 1.1}, "mixer": {"heads": 3, "dim": 4, "vdim": 5, "gate_cap": 8.0}}]}
    cfg.update(kw)
    return cfg


@pytest.mark.parametrize("rot", [{"dims": 8, "base": 500.0}, {"dims": 32, "base": 1e6, "scaling": {"factor": 5.0, "original": 300, "fast": 12.0, "slow": 2.0}},
                                 {"dims": 2, "base": 10.0, "scaling": {"factor": 2.0, "original": 7, "fast": 1.0, "slow": 1.0}}])
def test_rotary_table(rot):
    from applegpu_runtime_b200.rotary import rotary_table
    t = rotary_table(70, rot["dims"], rot["base"], rot.get("scaling"))
    x = np.zeros((70, rot["dims"]))
    x[:, 0::2] = 1.0                                          # (1, 0) turned by an angle is (cos, sin)
    want = R.rotate_pairs(x, np.arange(70), rot)
    assert np.max(np.abs(t[..., 0] - want[:, 0::2])) < 1e-7 and np.max(np.abs(t[..., 1] - want[:, 1::2])) < 1e-7


def test_yarn_keeps_fast_pairs_and_slows_slow_ones():
    rot = {"dims": 64, "base": 1e4, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}}
    f, amp = R.yarn_frequencies(rot)
    plain, _ = R.yarn_frequencies({"dims": 64, "base": 1e4})
    assert f[0] == plain[0] and math.isclose(f[-1], plain[-1] / 8.0) and math.isclose(amp, 0.1 * math.log(8.0) + 1.0)
    assert np.all(f <= plain) and np.all(f >= plain / 8.0 - 1e-12)


def test_safetensors_round_trip(tmp_path):
    from applegpu_runtime_b200.checkpoint import bf16_to_f32, f32_to_bf16, read_safetensors, write_safetensors
    rng = np.random.default_rng(0)
    a = rng.standard_normal((3, 5)).astype(np.float32)
    t = np.arange(6, dtype=np.int32).reshape(2, 3)
    write_safetensors(str(tmp_path / "m.safetensors"), {"a": a, "t": t})
    r = read_safetensors(str(tmp_path / "m.safetensors"))
    assert np.array_equal(r["t"], t) and r["t"].dtype == np.int32 and np.array_equal(r["a"], bf16_to_f32(f32_to_bf16(a)))
    torch = pytest.importorskip("torch")
    ties = np.array([1.00390625, 1.01171875, -1.00390625, 3e38, 1e-40], np.float32)
    assert np.array_equal(bf16_to_f32(f32_to_bf16(ties)), torch.from_numpy(ties).to(torch.bfloat16).float().numpy())


def test_packing():
    from applegpu_runtime_b200.seqmodel import interleaved, rows, side_by_side
    a, b = np.ones((3, 5), np.float32), 2 * np.ones((2, 5), np.float32)
    m = rows(a, b)
    assert m.shape == (5, 8) and np.all(m[:3, :5] == 1) and np.all(m[3:, :5] == 2) and np.all(m[:, 5:] == 0)
    m = rows(a, b, pad_rows=True)
    assert m.shape == (16, 8) and np.all(m[8:10, :5] == 2) and m.sum() == 15 + 20
    m = side_by_side(np.ones((4, 3), np.float32), 2 * np.ones((4, 6), np.float32))
    assert m.shape == (4, 16) and np.all(m[:, :3] == 1) and np.all(m[:, 3:8] == 0) and np.all(m[:, 8:14] == 2) and np.all(m[:, 14:] == 0)
    m = interleaved(np.arange(18, dtype=np.float32)[:, None], 100 + np.arange(18, dtype=np.float32)[:, None])
    assert m.shape == (64, 8) and m[:16, 0].tolist() == list(range(16)) and m[16:32, 0].tolist() == list(range(100, 116)) and m[32:34, 0].tolist() == [16, 17]
    assert m[48:50, 0].tolist() == [116, 117] and m[34:48].sum() == 0 and m[50:].sum() == 0
    with pytest.raises(ValueError):
        rows(a, np.ones((2, 4), np.float32))


def test_registry_and_shape_errors(gpu, tmp_path):
    from applegpu_runtime_b200 import models
    assert models.architecture_of(small_config()) == "Gedenex"
    assert models.architecture_of({"architectures": ["GPT2LMHeadModel"]}) == "GPT2LMHeadModel" and models.architecture_of({"model_type": "bert"}) == "bert"
    with pytest.raises(ValueError, match="unknown architecture"):
        models.build_model({"architecture": "Nobody"}, {})
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nobody"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        models.load_model(str(tmp_path))
    cfg = small_config()
    w = gpu.init_gedenex_weights(cfg)
    for name in ("l0.mix.uk", "loop.step", "l1.mlp.up"):
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            gpu.load_gedenex(cfg, {k: v for k, v in w.items() if k != name})
    with pytest.raises(ValueError, match="shape"):
        gpu.load_gedenex(cfg, {**w, "l1.mix.i": np.zeros((2, 22), np.float32)})
    bad = small_config()
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        gpu.load_gedenex(bad, w)


def test_layer_runs():
    cfg = small_config()
    assert R.layer_runs(cfg) == [(0, None, False), (1, 0, True), (1, 1, True)]
    assert R.layer_runs(small_config(loop=None)) == [(0, None, False), (1, None, False)]


def test_oracle_portions_agree(gpu):
    cfg = small_config()
    w = gpu.init_gedenex_weights(cfg, seed=1, std=0.4)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 14)
    want = R.forward(cfg, w, toks)
    states, got = [], []
    for lo, hi in ((0, 5), (5, 6), (6, 14)):
        got.append(R.forward(cfg, w, toks[lo:hi], states))
    assert np.max(np.abs(np.concatenate(got) - want)) < 1e-10


def test_oracle_mlstm_keeps_its_maximum_from_zero():
    """With quiet gates the normaliser's floor exp(-m) is what divides; m starts at 0."""
    q = k = np.full((1, 1, 2), 0.1)
    v = np.ones((1, 1, 2))
    o, (S, n, m) = R.mlstm_sequence(q, k, v, np.full((1, 1), -3.0), np.full((1, 1), -0.5))
    assert m[0] == -0.5
    w = math.exp(-2.5)
    assert np.allclose(o, w * 0.02 / (math.exp(0.5) + 1e-6)) and np.allclose(n, w * 0.1)
