"""Rurunex on the GPU against the plain float64 restatement in oracle/rurunex_ref.py: each mechanism alone, whole models,
portions, slots, batches, generation, command line and trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import rurunex_ref as R
from test_gpu_gedenex import bf16, close, put, rel, run_cuts

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 1e-4, "bfloat16": 9e-2}
DTYPES = ["float32", "bfloat16"]


def p8(n):
    return (n + 7) // 8 * 8


def padded(parts):
    """Column blocks [.., n] side by side, each padded with 7.0 to a multiple of 8 (what lies there must not matter)."""
    out = []
    for a in parts:
        b = np.full(a.shape[:-1] + (p8(a.shape[-1]),), 7.0, np.float32)
        b[..., :a.shape[-1]] = a
        out.append(b)
    return np.concatenate(out, axis=-1)


# ── norms and the feed-forward activation ───────────────────────────────────
@pytest.mark.parametrize("rows,width", [(1, 24), (5, 33), (40, 200), (3, 1024), (2, 9000)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_rms_add(gpu_dev, rows, width, dtype):
    rng = np.random.default_rng(rows + width)
    x, y = rng.standard_normal((2, rows, width)).astype(np.float32) * np.float32(0.3)
    post, w = 1 + rng.standard_normal((2, width)).astype(np.float32) * np.float32(0.3)
    g = gpu_dev
    gx = g.from_numpy(x)
    got = g.rms_add(gx, g.from_numpy(y), g.from_numpy(post), g.from_numpy(w), eps=2e-3, dtype=dtype).to_numpy()
    s = x + R.rms_norm(y.astype(np.float64), post, 2e-3)
    assert rel(gx.to_numpy(), s) < 1e-6
    assert rel(got, R.rms_norm(s, w, 2e-3)) < {"float32": 1e-6, "bfloat16": 4e-3}[dtype]


@pytest.mark.parametrize("rows,ff", [(1, 8), (7, 52), (33, 96), (5, 27)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_silu_glu(gpu_dev, rows, ff, dtype):
    gu = bf16(np.random.default_rng(ff).standard_normal((rows, 2 * ff)) * 3)
    gu[0, :3], gu[0, ff:ff + 3] = [60.0, -60.0, -400.0], [-50.0, 50.0, 50.0]
    got = gpu_dev.silu_glu(put(gpu_dev, gu, dtype)).to_numpy()
    want = R.silu(gu[:, :ff].astype(np.float64)) * gu[:, ff:]
    assert rel(got, want) < {"float32": 1e-6, "bfloat16": 4e-3}[dtype]


# ── matrix states with one decay per key channel ────────────────────────────
GLA = dict(delta=False, unit=False, softplus=False, gate_silu=True, taps=0, gr=0)
DELTA = dict(delta=True, unit=True, softplus=True, gate_silu=False, taps=4, gr=20)
KD_CASES = {
    "gla": dict(GLA, H=2, G=2, d=16, e=24, ar=16), "gla_odd": dict(GLA, H=3, G=3, d=20, e=13, ar=5), "gla_wide": dict(GLA, H=1, G=1, d=128, e=264, ar=24),
    "gla_192": dict(GLA, H=1, G=1, d=160, e=40, ar=8),
    "delta": dict(DELTA, H=2, G=2, d=32, e=32, ar=12), "delta_groups": dict(DELTA, H=6, G=2, d=24, e=40, ar=24, gr=9), "delta_odd": dict(DELTA, H=3, G=1, d=11, e=19, ar=3, gr=7, taps=2),
    "delta_128": dict(DELTA, H=1, G=1, d=128, e=128, ar=64, gr=64), "delta_96": dict(DELTA, H=2, G=1, d=72, e=80, ar=8), "delta_256": dict(DELTA, H=1, G=1, d=256, e=24, ar=8, taps=5),
    "delta_values_200": dict(DELTA, H=1, G=1, d=64, e=200, ar=8), "six_taps": dict(DELTA, H=2, G=1, d=40, e=24, ar=8, taps=6), "one_tap": dict(DELTA, H=2, G=1, d=16, e=16, ar=8, taps=1), "plain_delta": dict(DELTA, H=2, G=2, d=16, e=24, ar=8, unit=True, taps=0, gr=0, softplus=False),
    "conv_without_delta": dict(GLA, H=2, G=1, d=24, e=16, ar=8, taps=3, softplus=True, gr=6), "beyond_chunks": dict(DELTA, H=1, G=1, d=300, e=20, ar=8),
}


def kd_case(z, T, B, seed, decay=0.0, scale=1.0):
    """Inputs of a case; `decay` shifts the decays' inputs (towards forgetting for softplus, towards keeping otherwise)."""
    rng = np.random.default_rng(seed)
    H, G, d, e = z["H"], z["G"], z["d"], z["e"]
    c = dict(z, T=T, B=B, tau=5.0, eps=3e-5)
    n = lambda *s: bf16(rng.standard_normal(s) * scale)  # noqa: E731
    c["q"], c["k"], c["v"], c["a1"], c["g"] = n(B, T, G * d), n(B, T, G * d), n(B, T, H * e), n(B, T, z["ar"]), n(B, T, z["gr"] or H * e)
    c["beta"] = rng.standard_normal((B, T, H)).astype(np.float32)
    c["a2"], c["g2"] = bf16(rng.standard_normal((H * d, z["ar"])) * z["ar"] ** -0.5), bf16(rng.standard_normal((H * e, max(z["gr"], 1))) * max(z["gr"], 1) ** -0.5)
    c["bias"], c["rate"] = (rng.standard_normal(H * d) + decay).astype(np.float32), np.exp(rng.uniform(-2.0, 0.7, H)).astype(np.float32)
    c["norm"] = (1 + 0.2 * rng.standard_normal(e)).astype(np.float32)
    c["conv"] = (rng.standard_normal((2 * G * d + H * e, max(z["taps"], 1))) * 0.7).astype(np.float32)
    return c


def kd_want(c, b):
    """[T, H * e] and the state after the last token."""
    T, H, G, d, e = c["T"], c["H"], c["G"], c["d"], c["e"]
    parts, lo = [], 0
    for x in (c["q"][b], c["k"][b], c["v"][b]):
        x = x.astype(np.float64)
        if c["taps"]:
            w = c["conv"][lo:lo + x.shape[1]].astype(np.float64)
            x = R.silu(R.causal_conv(x, w, np.zeros((c["taps"] - 1, x.shape[1])))[0])
        parts.append(x)
        lo += x.shape[1]
    q, k, v = parts[0].reshape(T, G, d), parts[1].reshape(T, G, d), parts[2].reshape(T, H, e)
    if c["unit"]:
        q, k = R.unit(q), R.unit(k)
    q, k = np.repeat(q * d ** -0.5, H // G, axis=1), np.repeat(k, H // G, axis=1)
    zz = (c["a1"][b].astype(np.float64) @ c["a2"].T + c["bias"]).reshape(T, H, d)
    a = np.exp(-c["rate"][:, None] * R.softplus(zz) if c["softplus"] else R.log_sigmoid(zz) / c["tau"])
    S = np.zeros((H, d, e))
    if c["delta"]:
        o, S = R.delta_recurrence(q, k, v, a, R.sigmoid(c["beta"][b].astype(np.float64)), S)
    else:
        o, S = R.gla_recurrence(q, k, v, a, S)
    gate = c["g"][b].astype(np.float64)
    if c["gr"]:
        gate = gate @ c["g2"].T
    act = R.silu if c["gate_silu"] else R.sigmoid
    return R.rms_norm(o, c["norm"], c["eps"]).reshape(T, H * e) * act(gate), S


def kd_run(g, c, cuts, dtype, form):
    from applegpu_runtime_b200 import seqmodel as sm
    from applegpu_runtime_b200.seqmodel import rows
    flags = sum(f for f, on in ((sm.DELTA, c["delta"]), (sm.UNIT, c["unit"]), (sm.SOFTPLUS, c["softplus"]), (sm.GATE_SILU, c["gate_silu"])) if on)
    mem = g.key_decay_memory(c["B"], dtype, c["H"], c["G"], c["d"], c["e"], c["taps"])
    t = {n: g.from_numpy(c[n]) for n in ("bias", "norm", "rate")}
    a2, g2, conv = put(g, rows(c["a2"]), dtype), put(g, rows(c["g2"]), dtype), g.from_numpy(c["conv"].reshape(-1))
    out, lo = [], 0
    for n in cuts:
        s = slice(lo, lo + n)
        proj = padded([c[x][:, s] for x in ("q", "k", "v", "a1", "g")])
        y = g.key_decay(put(g, proj, dtype), a2, t["bias"], t["norm"], mem, g.from_numpy(np.full(c["B"], lo, np.int32)), c["H"], c["G"], c["d"], c["e"], c["ar"], c["gr"], flags, c["taps"],
                        c["tau"], c["eps"], beta=g.from_numpy(np.ascontiguousarray(c["beta"][:, s])) if c["delta"] else None, g2=g2 if c["gr"] else None,
                        rate=t["rate"] if c["softplus"] else None, conv=conv if c["taps"] else None, form=form)
        out.append(y.to_numpy())
        lo += n
    H, d, e = c["H"], c["d"], c["e"]
    return np.concatenate(out, axis=1), mem.to_numpy()[:, :H * d * e].reshape(c["B"], H, d, e)


@pytest.mark.parametrize("name", sorted(KD_CASES))
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", ["auto", "steps"])
def test_key_decay_portions(gpu_dev, name, dtype, form):
    """Two sequences in portions around the borders of chunks and blocks, state and convolution inputs carried along."""
    cuts = [2, 33, 1, 31, 64, 17, 1, 1, 2, 16, 45] if form == "auto" else [1, 2, 40, 16, 3]
    c = kd_case(KD_CASES[name], sum(cuts), 2, seed=len(name) + KD_CASES[name]["d"], decay=-1.0 if KD_CASES[name]["softplus"] else 2.0)
    got, S = kd_run(gpu_dev, c, cuts, dtype, form)
    for b in range(2):
        want, state = kd_want(c, b)
        assert rel(S[b], state) < {"float32": 2e-5, "bfloat16": 2e-4}[dtype]            # the state is float32 in either storage type
        assert rel(got[b], want) < {"float32": 1e-4, "bfloat16": 2e-2}[dtype]
    assert gpu_dev.pipeline_status() == 0


@pytest.mark.parametrize("kind", ["gla", "delta"])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("where", [0, 1, 7, 8, 15, 16, 31, 32, 63, 96, 288])
def test_key_decay_far_token(gpu_dev, kind, dtype, where):
    """One loud token under decays close to one comes back at the end of the portion, and reaches no row before itself."""
    z = dict(GLA if kind == "gla" else DELTA, H=2, G=2, d=48, e=32, ar=8, taps=0)
    T = 300
    c = kd_case(z, T, 1, seed=3, decay=9.0 if kind == "gla" else -9.0, scale=0.5)
    c["a1"] *= 0
    c["k"] *= 0.3 if kind == "gla" else 1.0
    u = np.zeros(z["d"], np.float32)
    u[5] = 9.0
    for h in range(2):
        s = slice(h * z["d"], (h + 1) * z["d"])
        c["k"][0, :, h * z["d"] + 5] = 0.0                     # nobody else writes along this direction
        c["k"][0, where, s], c["q"][0, T - 1, s] = u, u
    c["v"][0, where] *= 6.0
    c["beta"][0, where] = 6.0
    got, _ = kd_run(gpu_dev, c, [T], dtype, "auto")
    want, _ = kd_want(c, 0)
    assert rel(got[0], want) < {"float32": 1e-4, "bfloat16": 2e-2}[dtype]
    assert rel(got[0, -1], want[-1]) < {"float32": 1e-4, "bfloat16": 1e-2}[dtype]
    if where:
        c["k"][0, where:], c["v"][0, where:] = 5.0, -8.0
        again, _ = kd_run(gpu_dev, c, [T], dtype, "auto")
        assert np.array_equal(again[0, :where], got[0, :where])


@pytest.mark.parametrize("kind", ["gla", "delta"])
def test_key_decay_abrupt_forgetting(gpu_dev, kind):
    """Decays from one to nothing within a chunk: no factor may overflow or lose what the recurrence keeps."""
    z = dict(GLA if kind == "gla" else DELTA, H=2, G=1 if kind == "delta" else 2, d=32, e=24, ar=8, taps=0)
    c = kd_case(z, 200, 1, seed=11, decay=0.0)
    c["a1"] = bf16(np.random.default_rng(4).standard_normal(c["a1"].shape) * 60)
    got, S = kd_run(gpu_dev, c, [200], "bfloat16", "auto")
    want, state = kd_want(c, 0)
    assert np.all(np.isfinite(got)) and rel(S[0], state) < 2e-4 and close(got[0], want, 2e-2)


# ── grouped attention ───────────────────────────────────────────────────────
GA_SIZES = {
    "small": dict(H=2, G=1, d=16, e=8, pairs=8, window=0, cap=0.0), "odd": dict(H=6, G=3, d=20, e=13, pairs=7, window=37, cap=4.0),
    "tensor": dict(H=4, G=2, d=64, e=64, pairs=32, window=70, cap=6.0), "partly_turned": dict(H=3, G=3, d=48, e=40, pairs=12, window=64, cap=0.0),
    "wide": dict(H=2, G=1, d=128, e=128, pairs=64, window=129, cap=20.0), "many_heads": dict(H=20, G=1, d=24, e=16, pairs=12, window=0, cap=3.0),
    "values_256": dict(H=1, G=1, d=72, e=256, pairs=36, window=100, cap=9.0), "itself_only": dict(H=2, G=2, d=32, e=16, pairs=4, window=1, cap=2.0), "no_turn": dict(H=2, G=1, d=40, e=24, pairs=0, window=5, cap=0.0),
}


def ga_case(z, T, B, seed, max_len, loud=1.0):
    rng = np.random.default_rng(seed)
    c = dict(z, T=T, B=B, max_len=max_len, scale=1.4 * z["d"] ** -0.5 * loud, eps=2e-5)
    c["q"], c["k"], c["v"] = (bf16(rng.standard_normal((B, T, n))) for n in (z["H"] * z["d"], z["G"] * z["d"], z["G"] * z["e"]))
    c["qn"], c["kn"] = 1 + 0.3 * rng.standard_normal((2, z["d"])).astype(np.float32)
    c["rot"] = {"dims": 2 * z["pairs"], "base": 3000.0, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    return c


def ga_turned(c, x, heads, w, b):
    x = R.rms_norm(x[b].astype(np.float64).reshape(c["T"], heads, c["d"]), w, c["eps"])
    return R.rotate_halves(x, np.arange(c["T"]), c["rot"]) if c["pairs"] else x


def ga_want(c, b):
    q, k = ga_turned(c, c["q"], c["H"], c["qn"], b), ga_turned(c, c["k"], c["G"], c["kn"], b)
    v = c["v"][b].astype(np.float64).reshape(c["T"], c["G"], c["e"])
    return R.attention_rows(q, k, v, 0, c["scale"], c["cap"], c["window"]).reshape(c["T"], -1)


def ga_run(g, c, cuts, dtype, form, shared_with=None):
    """`shared_with`: (case, cuts) whose keys and values are used; its rows are appended ahead of each portion."""
    from applegpu_runtime_b200.rotary import rotary_table
    cache = put(g, np.full((c["B"], c["max_len"], p8(c["G"] * c["d"]) + p8(c["G"] * c["e"])), 50.0), dtype)       # rows never written must not matter
    rot = g.from_numpy(rotary_table(c["max_len"], 2 * c["pairs"], c["rot"]["base"], c["rot"]["scaling"])) if c["pairs"] else None
    out, lo = [], 0
    for n in cuts:
        s, pos = slice(lo, lo + n), g.from_numpy(np.full(c["B"], lo, np.int32))
        f = form if form != "mixed" else ("short" if n <= 16 else "portion")
        common = (rot, cache, pos, lo, c["H"], c["G"], c["d"], c["e"], c["scale"], c["cap"])
        proj = put(g, padded([c["q"][:, s], c["k"][:, s], c["v"][:, s]]), dtype)
        y = g.grouped_attention(proj, g.from_numpy(c["qn"]), g.from_numpy(c["kn"]), *common, window=c["window"], eps=c["eps"], form=f)
        if shared_with:
            o = shared_with
            proj = put(g, padded([o["q"][:, s]]), dtype)
            y = g.grouped_attention(proj, g.from_numpy(o["qn"]), None, *common, window=o["window"], shared=True, eps=c["eps"], form=f)
        out.append(y.to_numpy())
        lo += n
    return np.concatenate(out, axis=1)


def tensor_ok(z):
    return z["d"] % 8 == 0 and z["e"] % 8 == 0


@pytest.mark.parametrize("name", sorted(GA_SIZES))
@pytest.mark.parametrize("dtype", DTYPES)
def test_grouped_attention_forms_and_portions(gpu_dev, name, dtype):
    z, cuts = GA_SIZES[name], [3, 130, 1, 64, 2, 61]
    T = sum(cuts)
    c = ga_case(z, T, 2, 5, T + 3)
    want = [ga_want(c, b) for b in range(2)]
    for form in ["portion", "short", "mixed"] + (["tensor"] if dtype == "bfloat16" and tensor_ok(z) else []):
        got = ga_run(gpu_dev, c, cuts, dtype, form)
        for b in range(2):
            assert rel(got[b], want[b]) < {"float32": 3e-5, "bfloat16": 2e-2}[dtype], form
    assert gpu_dev.pipeline_status() == 0


@pytest.mark.parametrize("window", [1, 6, 90, 0])
@pytest.mark.parametrize("dtype", DTYPES)
def test_grouped_attention_shared_keys(gpu_dev, dtype, window):
    """Queries of another layer, with their own norm and window, over keys and values that are already cached."""
    cuts = [20, 1, 64, 2, 33]
    c = ga_case(dict(H=4, G=2, d=32, e=24, pairs=16, window=30, cap=5.0), sum(cuts), 2, 8, 130)
    o = dict(ga_case(dict(H=4, G=2, d=32, e=24, pairs=16, window=window, cap=5.0), sum(cuts), 2, 9, 130), k=c["k"], v=c["v"], kn=c["kn"])
    got = ga_run(gpu_dev, c, cuts, dtype, "mixed", shared_with=o)
    for b in range(2):
        assert rel(got[b], ga_want(o, b)) < {"float32": 3e-5, "bfloat16": 2e-2}[dtype]


@pytest.mark.parametrize("form", ["portion", "short", "tensor"])
@pytest.mark.parametrize("query,window", [(299, 64), (299, 65), (200, 128), (128, 129), (255, 1), (191, 63), (130, 127), (64, 300), (70, 7)])
def test_grouped_attention_window_edges(gpu_dev, form, query, window):
    """The last key inside a row's window can win the row; the one just outside, and the one just after the row, change nothing."""
    z, T = dict(H=2, G=1, d=64, e=32, pairs=16, window=window, cap=0.0), 300
    c = ga_case(z, T, 1, 21, T, loud=4.0)
    inside = max(0, query - window + 1)
    k = ga_turned(c, c["k"], 1, c["kn"], 0)[:, 0]
    # a query that turns into the direction of the key at `inside`
    turn = R.rotate_halves(np.eye(64)[:, None], np.full(64, query), c["rot"])[:, 0]       # row i: image of unit vector i
    for h in range(2):
        c["q"][0, query, h * 64:(h + 1) * 64] = bf16((turn @ k[inside]) / c["qn"])
    got = ga_run(gpu_dev, c, [T], "bfloat16", form)[0]
    want = ga_want(c, 0)
    assert rel(got[query], want[query]) < 2e-2 and rel(got, want) < 3e-2
    if window > 1:
        row = want[query].reshape(2, 32) - c["v"][0, inside]
        assert np.max(np.abs(row)) < 0.2 * np.max(np.abs(c["v"][0, inside]))              # it does win
    for other in ([query - window] if query >= window else []) + ([query + 1] if query + 1 < T else []):
        m = dict(c, k=c["k"].copy(), v=c["v"].copy())
        m["k"][0, other], m["v"][0, other] = m["k"][0, inside], 90.0
        assert np.array_equal(ga_run(gpu_dev, m, [T], "bfloat16", form)[0, query], got[query])


# ── models ──────────────────────────────────────────────────────────────────
YARN = {"factor": 6.0, "original": 48, "fast": 16.0, "slow": 1.0}


def att(H, G, d, e, window, dims=None, source=None, base=2000.0, scaling=YARN, cap=6.0):
    rot = {"dims": dims or d, "base": base}
    if scaling:
        rot["scaling"] = scaling
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": e, "mask": {"size": window} if window else None, "rot": rot, "scale": 1.3 * d ** -0.5, "softcap": cap}
    if source is not None:
        m["kv_from"] = source
    return ("attention", m)


def gla(H, d, e, tau=6.0):
    return ("gla", {"heads": H, "dim": d, "vdim": e, "tau": tau})


def delta(H, G, d, e, conv=4):
    return ("channel_delta", {"heads": H, "kv_heads": G, "dim": d, "vdim": e, "conv": conv})


def config(width, layers, vocab=130, eps=3e-5, scale=3.7, logit_scale=0.8):
    return {"architecture": "Rurunex", "embedding": {"scale": scale}, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}


CONFIGS = {
    "mixed": config(96, [(gla(3, 16, 24), 72), (att(4, 2, 24, 16, 40), None), (delta(4, 2, 24, 16), 56), (att(4, 2, 24, 16, 11, source=1), 40), (att(4, 2, 24, 16, 70, source=1), None)]),
    "odd_sizes": config(75, [(delta(3, 1, 10, 13, conv=3), 37), (att(6, 3, 14, 9, 19, dims=6, scaling=None), 50), (gla(1, 7, 22), None), (att(6, 3, 14, 9, 33, dims=6, source=1, scaling=None), None)],
                        vocab=101, scale=1.0, logit_scale=1.0),
    "no_caps": config(64, [(att(2, 2, 32, 32, None, cap=None), 64), (delta(2, 2, 32, 64, conv=2), None)], vocab=77),
    "wide_heads": config(128, [(gla(1, 128, 136), 64), (delta(1, 1, 128, 128), None), (att(2, 1, 128, 128, 65), 128)]),
}


def weights(cfg, seed=3):
    """Weights loud enough that every mechanism shows in the logits, rounded to bfloat16."""
    from applegpu_runtime_b200 import init_rurunex_weights
    rng = np.random.default_rng(seed)
    w = {}
    for name, a in init_rurunex_weights(cfg, seed, ranks={"gla": 11, "channel_delta": 12}).items():
        if name.endswith(".conv"):
            a = rng.standard_normal(a.shape) * 0.8
        elif name == "embed":
            a = a / 0.02 * 0.7
        elif a.ndim == 2:
            a = a / 0.02 * a.shape[1] ** -0.5
        elif name.endswith("a2.b"):
            a = 3.0 + 1.5 * rng.standard_normal(a.shape)
        elif name.endswith("dt_bias"):
            a = -3.0 + 1.5 * rng.standard_normal(a.shape)
        elif name.endswith("A_log"):
            a = rng.uniform(-1.0, 1.0, a.shape)
        else:
            a = a + 0.3 * rng.standard_normal(a.shape)         # unit weights and differences from one alike
        w[name] = bf16(a)
    return w


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_model_layers_portions_slots(gpu_dev, name, dtype):
    cfg, g = CONFIGS[name], gpu_dev
    w = weights(cfg)
    model = g.load_rurunex(cfg, w, dtype)
    T = 150
    toks = np.random.default_rng(8).integers(0, cfg["vocab"], T).tolist()
    trace = []
    want = R.forward(cfg, w, toks, trace=trace)
    eng = model.engine(slots=3, max_len=T + 10)
    _, _, layers = eng.forward(toks, want=[], logits=False, layers=True)
    assert layers.shape[0] == len(trace)
    for got, ref in zip(layers, trace):
        assert close(got, ref, TOL[dtype])
    for slot, cuts in [(1, [T]), (2, [2] * 75), (1, [1] * T), (0, [17, 2, 3, 64, 31, 1, 1, 1, 16, 14]), (2, [16, 17, 100, 2, 15])]:
        eng.reset(slot)                                        # also slots that held other things before
        assert eng.length(slot) == 0
        got = run_cuts(eng, toks, cuts, slot)
        assert close(got, want, TOL[dtype]), (slot, cuts[:4])
        assert eng.length(slot) == T
    _, _, one = eng.forward(toks[:1], slot=0 if eng.reset(0) is None else 0, want=[], logits=False, layers=True)
    assert close(one, np.stack([t[:1] for t in trace]), TOL[dtype])
    with pytest.raises(ValueError):
        eng.forward(toks[:11], slot=2)                         # outgrows the slot; the slot is left as it was
    assert eng.length(2) == T
    with pytest.raises(ValueError):
        eng.forward([cfg["vocab"]], slot=0)
    eng.close()
    assert g.pipeline_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(gpu_dev, dtype):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, 5)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 330).tolist()
    want = R.forward(cfg, w, toks)
    eng = gpu_dev.load_rurunex(cfg, w, dtype).engine(1, 330)
    got = run_cuts(eng, toks, [20] + [1] * 310)
    assert eng.uses_graph
    assert close(got, want, TOL[dtype])


def test_batch_against_alone(gpu_dev):
    """Sequences of unequal lengths decoded together give what each gives alone; equal ones as one portion likewise."""
    cfg = CONFIGS["mixed"]
    model = gpu_dev.load_rurunex(cfg, weights(cfg), "float32")
    rng = np.random.default_rng(4)
    prompts = [rng.integers(0, cfg["vocab"], n).astype(np.int32) for n in (5, 70, 1, 33)]
    more = rng.integers(0, cfg["vocab"], (4, 12)).astype(np.int32)
    eng, alone = model.engine(4, 100), model.engine(1, 100)
    for i, p in enumerate(prompts):
        eng.forward(p, slot=i, logits=False)
    joint = np.stack([eng.forward(more[:, t:t + 1])[0] for t in range(6)], axis=1)
    joint = np.concatenate([joint, eng.forward(more[:, 6:], want=[s * 6 + t for s in range(4) for t in range(6)])[0].reshape(4, 6, -1)], axis=1)   # 24 rows of short portions
    for i, p in enumerate(prompts):
        alone.reset(0)
        alone.forward(p, logits=False)
        assert rel(joint[i], run_cuts(alone, more[i].tolist(), [1] * 12)) < 2e-5
    same = rng.integers(0, cfg["vocab"], (4, 40)).astype(np.int32)
    for dtype in DTYPES:
        m = model if dtype == "float32" else gpu_dev.load_rurunex(cfg, weights(cfg), dtype)
        eng, alone = m.engine(4, 100), m.engine(1, 100)
        eng.forward(same[2:, :20], slot=2, logits=False)       # two of the four hold something already
        both = eng.forward(same)[0]
        for i in range(4):
            alone.reset(0)
            if i >= 2:
                alone.forward(same[i, :20], logits=False)
            assert rel(both[i], alone.forward(same[i])[0][0]) < {"float32": 2e-5, "bfloat16": 2e-2}[dtype]


def test_portions_longer_than_a_step(gpu_dev):
    """A prompt with more rows than one step takes: the engine cuts it itself."""
    cfg = config(32, [(gla(1, 16, 16), None), (att(2, 1, 16, 16, 100, base=1e5), 32), (delta(2, 1, 16, 16), None)], vocab=60)
    toks = np.random.default_rng(3).integers(0, 60, 8300).tolist()
    eng = gpu_dev.load_rurunex(cfg, weights(cfg, 21), "bfloat16").engine(1, 8300)
    rows = [0, 17, 5000, 8191, 8192, 8193, 8299]
    once = eng.forward(toks, want=rows)[0]
    eng.reset(0)
    parts, lo = [], 0
    for n in (3001, 1, 4100, 1198):
        parts.append(eng.forward(toks[lo:lo + n], want=[r - lo for r in rows if lo <= r < lo + n])[0])
        lo += n
    assert rel(once, np.concatenate(parts)) < TOL["bfloat16"]
    assert gpu_dev.pipeline_status() == 0


def test_more_sequences_than_step_rows(gpu_dev):
    """Eighteen sequences: the linears of a step go to the GEMM, the mixers stay token by token."""
    from applegpu_runtime_b200.generate import greedy_generate
    cfg = CONFIGS["mixed"]
    model = gpu_dev.load_rurunex(cfg, weights(cfg, 9), "float32")
    prompts = [np.random.default_rng(i).integers(0, cfg["vocab"], 3 + i).tolist() for i in range(18)]
    out = greedy_generate(model, prompts, 6)
    for i in (0, 7, 17):
        assert greedy_generate(model, [prompts[i]], 6)[0].tolist() == out[i]


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(gpu_dev, dtype):
    from applegpu_runtime_b200.generate import generate, greedy_generate
    cfg = CONFIGS["mixed"]
    w = weights(cfg, 9)
    model = gpu_dev.build_model(cfg, w, dtype)
    rng = np.random.default_rng(6)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (19, 3, 40)]
    out = greedy_generate(model, prompts, 10)
    assert model.last_decode_stats["graph"]
    assert greedy_generate(model, prompts, 10, engine="direct") == out
    for p, o in zip(prompts, out):
        assert o[:len(p)] == p and len(o) == len(p) + 10
        logits = R.forward(cfg, w, o[:-1])[len(p) - 1:]
        if dtype == "float32":
            assert logits.argmax(-1).tolist() == o[len(p):]
        else:                                                  # a choice may differ where two logits are within rounding
            took = logits[np.arange(10), o[len(p):]]
            assert np.all(logits.max(-1) - took < 0.1 * np.std(logits))
        assert generate(model, p, 10, temperature=0) == o
    sampled = generate(model, prompts[1], 5, temperature=1.0)
    assert len(sampled) == 8 and all(0 <= t < cfg["vocab"] for t in sampled)


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    from applegpu_runtime_b200.checkpoint import write_safetensors
    cfg = CONFIGS["odd_sizes"]
    d = tmp_path_factory.mktemp("model")
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(d / "model.safetensors"), weights(cfg, 12))
    return d


def test_command_line(gpu_dev, folder):
    cfg, w = CONFIGS["odd_sizes"], weights(CONFIGS["odd_sizes"], 12)
    r = subprocess.run([sys.executable, "-m", "applegpu_runtime_b200", "generate", "--model", str(folder), "--dtype", "float32", "--prompt", "4,9,17", "--prompt", "8",
                        "--max-tokens", "6"], cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    got = [json.loads(x) for x in r.stdout.splitlines()]
    for p, o in zip([[4, 9, 17], [8]], got):
        assert o[:len(p)] == p
        assert R.forward(cfg, w, o[:-1])[len(p) - 1:].argmax(-1).tolist() == o[len(p):]


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(gpu_dev, folder, tmp_path, dtype):
    cfg, w = CONFIGS["odd_sizes"], weights(CONFIGS["odd_sizes"], 12)
    rng = np.random.default_rng(1)
    a, b = rng.integers(0, cfg["vocab"], 60).tolist(), rng.integers(0, cfg["vocab"], 21).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}], "end": []}, {"step": 1, "entries": [{"id": "a", "tokens": a[50:52], "want": []}], "end": []}]
    steps += [{"step": 2 + i, "entries": [{"id": "a", "tokens": [a[52 + i]], "want": [0]}], "end": ["a"] if i == 7 else []} for i in range(8)]
    steps += [{"step": 10, "entries": [{"id": "b", "tokens": b, "want": [20, 3]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "64"], cwd=ROOT,
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(11)]
    wa, wb = R.forward(cfg, w, a), R.forward(cfg, w, b)
    want = {0: wa[[0, 49]], **{2 + i: wa[[52 + i]] for i in range(8)}, 10: wb[[20, 3]]}
    for i, ref in want.items():
        assert rel(np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]), ref) < TOL[dtype]
