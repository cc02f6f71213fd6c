"""Gedenex on the GPU against the plain float64 restatement in oracle/gedenex_ref.py: each mechanism alone, whole models,
portions, slots, batches, generation, command line and trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import gedenex_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}


def bf16(x):
    from applegpu_runtime_b200.checkpoint import bf16_to_f32, f32_to_bf16
    return bf16_to_f32(f32_to_bf16(np.ascontiguousarray(x, np.float32)))


def put(g, x, dtype):
    t = g.from_numpy(np.ascontiguousarray(x, np.float32))
    if dtype != "float32":
        t = g.cast(t, dtype)
        t.eval()
    return t


def rel(got, want):
    return float(np.max(np.abs(got - want)) / max(np.max(np.abs(want)), 1e-6))


def close(got, want, lim):
    """Every row within `lim` of the largest value. In bfloat16 one row in twenty may miss it: where a head's read-out nearly
    cancels, its norm blows the rounding of q and k up to full size."""
    err = np.max(np.abs(got - want), axis=-1).reshape(-1) / max(np.max(np.abs(want)), 1e-6)
    return np.mean(err > lim) <= (0.05 if lim > 1e-3 else 0.0)


# ── mechanisms ──────────────────────────────────────────────────────────────
@pytest.mark.parametrize("rows,width", [(1, 24), (5, 33), (40, 200), (3, 1024), (2, 9000)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_rms_norm(gpu_dev, rows, width, dtype):
    rng = np.random.default_rng(rows + width)
    x, w = rng.standard_normal((rows, width)).astype(np.float32) * 1e-2, rng.standard_normal(width).astype(np.float32)
    got = gpu_dev.rms_norm(gpu_dev.from_numpy(x), gpu_dev.from_numpy(w), eps=3e-4, dtype=dtype).to_numpy()
    assert rel(got, R.rms_norm(x.astype(np.float64), w, 3e-4)) < {"float32": 1e-6, "bfloat16": 4e-3}[dtype]


@pytest.mark.parametrize("rows,ff", [(1, 8), (7, 52), (33, 96), (5, 27)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_clamped_glu(gpu_dev, rows, ff, dtype):
    rng = np.random.default_rng(ff)
    gu = bf16(rng.standard_normal((rows, 2 * ff)) * 3)
    gu[0, 0], gu[0, ff], gu[0, 1], gu[0, ff + 1] = 50.0, -50.0, -400.0, 50.0       # both clamps, and no lower clamp on the gate
    got = gpu_dev.clamped_glu(put(gpu_dev, gu, dtype), 2.25).to_numpy()
    want = R.clamped_glu(gu[:, :ff].astype(np.float64), gu[:, ff:].astype(np.float64), 2.25)
    assert rel(got, want) < {"float32": 1e-6, "bfloat16": 4e-3}[dtype]


def mlstm_case(T, H, d, e, seed, B=1, forget=2.0, scale=1.0):
    rng = np.random.default_rng(seed)
    proj = bf16(rng.standard_normal((B, T, 2 * H * (d + e))) * scale)
    gates = (rng.standard_normal((B, T, 2 * H)) * 2.0).astype(np.float32)
    bias = np.concatenate([rng.standard_normal(H), forget + rng.standard_normal(H)]).astype(np.float32)
    norm = (1.0 + 0.2 * rng.standard_normal(H * e)).astype(np.float32)
    return proj, gates, bias, norm


def mlstm_want(proj, gates, bias, norm, H, d, e, cap, eps, state=None):
    T = proj.shape[0]
    p = proj.astype(np.float64)
    q = p[:, :H * d].reshape(T, H, d) * d ** -0.5
    k = p[:, H * d:2 * H * d].reshape(T, H, d)
    v = p[:, 2 * H * d:2 * H * d + H * e].reshape(T, H, e)
    z = p[:, 2 * H * d + H * e:2 * H * (d + e)]
    raw = gates.astype(np.float64) + bias
    li, lf = cap * np.tanh(raw[:, :H] / cap), R.log_sigmoid(cap * np.tanh(raw[:, H:] / cap))
    o, state = R.mlstm_sequence(q, k, v, li, lf, state)
    return R.head_norm(o, eps).reshape(T, H * e) * norm * R.sigmoid(z), state


def state_parts(s, H, d, e):
    return s[:H * d * e].reshape(H, d, e), s[H * d * e:H * d * e + H * d].reshape(H, d), s[H * d * e + H * d:H * d * e + H * d + H]


MLSTM_SIZES = [(1, 16, 16), (3, 20, 28), (2, 64, 128), (2, 8, 37), (1, 128, 256), (2, 72, 96), (2, 200, 40), (1, 24, 264), (1, 136, 520)]


@pytest.mark.parametrize("H,d,e", MLSTM_SIZES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("form", ["chunked", "simple", "steps"])
def test_mlstm_portions(gpu_dev, H, d, e, dtype, form):
    """Two sequences in portions around the borders of chunks and tiles, state carried from portion to portion."""
    cuts = [2, 63, 1, 65, 130, 59, 257] if form != "steps" else [1, 2, 16, 5]
    T, B, cap, eps = sum(cuts), 2, 9.0, 2e-5
    proj, gates, bias, norm = mlstm_case(T, H, d, e, seed=H * d + e, B=B)
    n = (H * (d * e + d + 1) + 3) // 4 * 4
    g = gpu_dev
    state = g.from_numpy(np.zeros((B, n), np.float32))
    bt, nt = g.from_numpy(bias), g.from_numpy(norm)
    out, lo = [], 0
    for c in cuts:
        out.append(g.mlstm(put(g, proj[:, lo:lo + c], dtype), g.from_numpy(gates[:, lo:lo + c]), bt, nt, state, H, d, e, cap, eps, form=form).to_numpy())
        lo += c
    got, st = np.concatenate(out, axis=1), state.to_numpy()
    for b in range(B):
        want, (S, nn, m) = mlstm_want(proj[b], gates[b], bias, norm, H, d, e, cap, eps)
        assert rel(got[b], want) < {"float32": 1e-4, "bfloat16": 2e-2}[dtype]
        gS, gn, gm = state_parts(st[b], H, d, e)
        assert rel(gS, S) < 2e-4 and rel(gn, nn) < 2e-4 and np.max(np.abs(gm - m)) < 1e-4       # the state is float32 in either storage type
    assert g.pipeline_status() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("where", [0, 1, 63, 64, 127, 128, 255, 256, 399])
def test_mlstm_far_token(gpu_dev, dtype, where):
    """One loud token under nearly open forget gates: its value must come back at the end of the portion, wherever it lies."""
    T, H, d, e, cap = 400, 2, 64, 64, 15.0
    proj, gates, bias, norm = mlstm_case(T, H, d, e, seed=5)
    gates[:], bias[:H], bias[H:] = 0.0, -4.0, 14.0
    u = np.zeros(d, np.float32)
    u[3] = 6.0
    for h in range(H):
        proj[0, where, H * d + h * d:H * d + (h + 1) * d] = u
        proj[0, T - 1, h * d:(h + 1) * d] = u
    gates[0, where, :H] = 12.0
    g = gpu_dev
    state = g.from_numpy(np.zeros((1, (H * (d * e + d + 1) + 3) // 4 * 4), np.float32))
    got = g.mlstm(put(g, proj, dtype), g.from_numpy(gates), g.from_numpy(bias), g.from_numpy(norm), state, H, d, e, cap).to_numpy()[0]
    want, _ = mlstm_want(proj[0], gates[0], bias, norm, H, d, e, cap, 1e-5)
    assert rel(got[-1], want[-1]) < {"float32": 1e-4, "bfloat16": 1e-2}[dtype]
    assert rel(got, want) < {"float32": 1e-4, "bfloat16": 2e-2}[dtype]
    if where:
        # the token itself must not reach rows before it
        proj2 = proj.copy()
        proj2[0, where:] += 7.0
        state = g.from_numpy(np.zeros((1, (H * (d * e + d + 1) + 3) // 4 * 4), np.float32))
        again = g.mlstm(put(g, proj2, dtype), g.from_numpy(gates), g.from_numpy(bias), g.from_numpy(norm), state, H, d, e, cap).to_numpy()[0]
        assert np.array_equal(again[:where], got[:where])


LATENT_SIZES = [dict(H=1, d=8, rd=8, e=8, r=8), dict(H=3, d=20, rd=12, e=28, r=40), dict(H=2, d=64, rd=64, e=64, r=64), dict(H=4, d=24, rd=16, e=40, r=136),
                dict(H=2, d=128, rd=64, e=128, r=512), dict(H=9, d=16, rd=32, e=136, r=72), dict(H=1, d=192, rd=64, e=256, r=96), dict(H=2, d=40, rd=6, e=20, r=33)]


def latent_case(g, T, B, z, dtype, seed, max_len, base=5000.0, scaling=None):
    from applegpu_runtime_b200.rotary import rotary_table
    from applegpu_runtime_b200.seqmodel import rows
    rng = np.random.default_rng(seed)
    cols = z["H"] * (z["d"] + z["rd"]) + z["r"] + z["rd"]
    c = dict(z, B=B, max_len=max_len, dtype=dtype)
    c["proj"] = bf16(rng.standard_normal((B, T, (cols + 7) // 8 * 8)))
    c["norm"] = (1 + 0.1 * rng.standard_normal(z["r"])).astype(np.float32)
    c["uk"] = bf16(rng.standard_normal((z["H"] * z["d"], z["r"])) * z["r"] ** -0.5)
    c["uv"] = bf16(rng.standard_normal((z["H"] * z["e"], z["r"])) * z["r"] ** -0.5)
    c["rot"] = {"dims": z["rd"], "base": base, **({"scaling": scaling} if scaling else {})}
    c["scale"] = 1.3 * (z["d"] + z["rd"]) ** -0.5
    c["t"] = dict(norm=g.from_numpy(c["norm"]), up=put(g, rows(c["uk"], c["uv"], pad_rows=True), dtype), rot=g.from_numpy(rotary_table(max_len, z["rd"], base, scaling)))
    return c


def new_cache(g, c):
    p8 = lambda n: (n + 7) // 8 * 8  # noqa: E731
    return put(g, np.full((c["B"], c["max_len"], p8(c["r"]) + p8(c["rd"])), 3.0), c["dtype"])      # rows that were never written must not matter


def latent_run(g, c, lo, hi, cache, form):
    pos = g.from_numpy(np.full(c["B"], lo, np.int32))
    return g.latent_attention(put(g, c["proj"][:, lo:hi], c["dtype"]), c["t"]["norm"], c["t"]["up"], c["t"]["rot"], cache, pos, lo, c["H"], c["d"], c["rd"], c["e"], c["r"],
                              c["scale"], 1e-5, form).to_numpy()


def latent_want(c, b, T):
    w = {"q": None}
    H, d, rd, r = c["H"], c["d"], c["rd"], c["r"]
    nq = H * (d + rd)
    # the mixer of the oracle with identity projections: its input is the projection row itself
    cols = c["proj"].shape[2]
    sel = np.eye(cols)
    w = {"q": sel[:nq], "dkv": sel[nq:nq + r + rd], "dkv.norm": c["norm"], "uk": c["uk"], "uv": c["uv"], "o": np.eye(H * c["e"])}
    mixer = dict(heads=H, dim=d, rot_dim=rd, vdim=c["e"], kv_rank=r, scale=c["scale"], rot=c["rot"])
    return R.latent_attention_mixer(c["proj"][b, :T].astype(np.float64), {k: np.asarray(v, np.float64) for k, v in w.items()}, "", mixer, 1e-5)[0]


@pytest.mark.parametrize("size", range(len(LATENT_SIZES)))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_latent_attention_forms_and_portions(gpu_dev, size, dtype):
    g, z = gpu_dev, LATENT_SIZES[size]
    cuts, B = [3, 130, 1, 64, 127], 2
    T = sum(cuts)
    c = latent_case(g, T, B, z, dtype, 10 + size, T + 5, scaling={"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0} if size % 2 else None)
    want = [latent_want(c, b, T) for b in range(B)]
    lim = {"float32": 3e-5, "bfloat16": 2e-2}[dtype]
    tensor = dtype == "bfloat16" and not any(z[k] % 8 for k in ("d", "rd", "e"))
    for form in ["expanded", "latent", "mixed"] + (["tensor"] if tensor else []):
        cache, lo, out = new_cache(g, c), 0, []
        for n in cuts:
            f = form if form != "mixed" else ("latent" if n < 16 else "expanded")
            out.append(latent_run(g, c, lo, lo + n, cache, f))
            lo += n
        got = np.concatenate(out, axis=1)
        for b in range(B):
            assert rel(got[b], want[b]) < lim, form
    assert g.pipeline_status() == 0


@pytest.mark.parametrize("form", ["expanded", "latent", "tensor"])
@pytest.mark.parametrize("key,query", [(0, 299), (63, 299), (64, 128), (127, 128), (128, 128), (191, 255), (255, 256), (200, 201), (299, 299)])
def test_latent_attention_far_key(gpu_dev, form, key, query):
    """A key that dominates one query: the query must return that token's value, and a loud key just after a query must not
    reach it."""
    g, z = gpu_dev, dict(H=2, d=64, rd=16, e=48, r=64)
    T, d, rd = 300, 64, 16
    c = latent_case(g, T, 1, z, "bfloat16", 77, T, base=1e6)
    c["rot"]["base"] = 1e6
    c["proj"] *= 0.3
    H, nq = z["H"], z["H"] * (d + rd)
    # unrotated part: queries along the key's own direction
    lat = c["proj"][0, key, nq:nq + 64].astype(np.float64)
    cn = R.rms_norm(lat, c["norm"], 1e-5)
    for h in range(H):
        kd = c["uk"][h * d:(h + 1) * d].astype(np.float64) @ cn
        c["proj"][0, query, h * (d + rd):h * (d + rd) + d] = bf16(kd * 60.0 / (np.linalg.norm(kd) ** 2 * c["scale"]))
    got = latent_run(g, c, 0, T, new_cache(g, c), form)[0]
    want = latent_want(c, 0, T)
    assert rel(got[query], want[query]) < 1e-2 and rel(got, want) < 2e-2
    if query + 1 < T:
        loud = {k: v for k, v in c.items()}
        loud["proj"] = c["proj"].copy()
        loud["proj"][0, query + 1:, nq:] *= 40.0
        again = latent_run(g, loud, 0, T, new_cache(g, c), form)[0]
        assert np.array_equal(again[:query + 1], got[:query + 1])


# ── models ──────────────────────────────────────────────────────────────────
def ml(H, d, e, cap=11.0):
    return {"heads": H, "dim": d, "vdim": e, "gate_cap": cap}


def la(H, d, rd, e, r, base=2000.0, scaling=None):
    rot = {"dims": rd, "base": base}
    if scaling:
        rot["scaling"] = scaling
    return {"heads": H, "dim": d, "rot_dim": rd, "vdim": e, "kv_rank": r, "scale": 0.17, "rot": rot}


def config(width, layers, loop=None, vocab=130, eps=3e-5):
    return {"architecture": "Gedenex", "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff[0], "limit": ff[1]}} for t, m, ff in layers],
            "loop": loop, "norm": {"eps": eps}, "vocab": vocab, "width": width}


YARN = {"factor": 6.0, "original": 48, "fast": 16.0, "slow": 1.0}
CONFIGS = {
    "looped": config(96, [("latent_attention", la(3, 16, 8, 24, 40, scaling=YARN), (72, 1.25)), ("mlstm", ml(2, 24, 40), (56, 2.0)), ("mlstm", ml(3, 16, 16), (40, 0.75))],
                     loop={"start": 1, "stop": 3, "times": 3}),
    "odd_sizes": config(75, [("mlstm", ml(3, 10, 13), (37, 1.5)), ("latent_attention", la(5, 11, 6, 9, 21), (50, 1.1)), ("mlstm", ml(1, 7, 22), None)],
                        loop={"start": 0, "stop": 2, "times": 2}, vocab=101),
    "no_loop_no_mlp": config(64, [("latent_attention", la(2, 32, 32, 32, 64), None), ("mlstm", ml(4, 16, 32), None)], vocab=77),
    "wide_heads": config(128, [("mlstm", ml(1, 128, 256), (64, 7.0)), ("latent_attention", la(1, 136, 64, 128, 256, scaling=YARN), (128, 7.0))], loop={"start": 0, "stop": 1, "times": 1}),
}


def weights(cfg, seed=3):
    """Weights loud enough that every mechanism shows in the logits, rounded to bfloat16."""
    from applegpu_runtime_b200 import init_gedenex_weights
    rng = np.random.default_rng(seed)
    w = {}
    for name, a in init_gedenex_weights(cfg, seed).items():
        if a.ndim == 2 and name not in ("embed", "loop.step"):
            a = a / 0.02 * a.shape[1] ** -0.5
        elif name in ("embed", "loop.step"):
            a = a / 0.02 * 0.7
        elif name.endswith(".i.b"):
            a = rng.standard_normal(a.shape)
        elif name.endswith(".f.b"):
            a = 2.0 + 1.5 * rng.standard_normal(a.shape)
        else:
            a = 1.0 + 0.3 * rng.standard_normal(a.shape)
        w[name] = bf16(a)
    return w


def run_cuts(eng, toks, cuts, slot=0):
    out, lo = [], 0
    for c in cuts:
        out.append(eng.forward(toks[lo:lo + c], slot=slot, want=list(range(c)))[0])
        lo += c
    assert lo == len(toks)
    return np.concatenate(out)


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_model_layers_portions_slots(gpu_dev, name, dtype):
    cfg, g = CONFIGS[name], gpu_dev
    w = weights(cfg)
    model = g.load_gedenex(cfg, w, dtype)
    T = 150
    rng = np.random.default_rng(8)
    toks = rng.integers(0, cfg["vocab"], T).tolist()
    trace = []
    want = R.forward(cfg, w, toks, trace=trace)
    eng = model.engine(slots=3, max_len=T + 10)
    lim = TOL[dtype] * 3
    _, _, layers = eng.forward(toks, want=[], logits=False, layers=True)
    assert layers.shape[0] == len(trace)
    for got, ref in zip(layers, trace):
        assert close(got, ref, lim)
    for slot, cuts in [(1, [T]), (2, [2] * 75), (1, [1] * T), (0, [17, 2, 3, 64, 31, 1, 1, 1, 16, 14]), (2, [16, 17, 100, 2, 15])]:
        eng.reset(slot)                                        # also slots that held other things before
        assert eng.length(slot) == 0
        got = run_cuts(eng, toks, cuts, slot)
        assert close(got, want, lim), (slot, cuts[:4])
        assert eng.length(slot) == T
    with pytest.raises(ValueError):
        eng.forward(toks[:11], slot=2)                         # outgrows the slot; the slot is left as it was
    assert eng.length(2) == T
    with pytest.raises(ValueError):
        eng.forward([cfg["vocab"]], slot=0)
    eng.close()
    assert g.pipeline_status() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(gpu_dev, dtype):
    cfg = CONFIGS["looped"]
    w = weights(cfg, 5)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 330).tolist()
    want = R.forward(cfg, w, toks)
    eng = gpu_dev.load_gedenex(cfg, w, dtype).engine(1, 330)
    got = run_cuts(eng, toks, [20] + [1] * 310)
    assert eng.uses_graph
    assert close(got, want, TOL[dtype] * 3)


def test_batch_against_alone(gpu_dev):
    """Sequences of unequal lengths decoded together give what each gives alone."""
    cfg, g = CONFIGS["looped"], gpu_dev
    w = weights(cfg)
    model = g.load_gedenex(cfg, w, "float32")
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
        got = run_cuts(alone, more[i].tolist(), [1] * 12)
        assert rel(joint[i], got) < 1e-5
    # equal lengths as one step, more rows than the step kernels take
    same = rng.integers(0, cfg["vocab"], (4, 40)).astype(np.int32)
    eng.reset(0, 4)
    both = eng.forward(same)[0]
    for i in range(4):
        alone.reset(0)
        assert rel(both[i], alone.forward(same[i])[0][0]) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_longer_than_a_step(gpu_dev, dtype):
    """A prompt, and a batch of prompts, with more rows than one step takes: the engine cuts them itself."""
    cfg = config(32, [("mlstm", ml(1, 16, 16), None), ("latent_attention", la(1, 16, 8, 16, 24, base=1e5), (32, 2.0))], vocab=60)
    w = weights(cfg, 21)
    rng = np.random.default_rng(3)
    model = gpu_dev.load_gedenex(cfg, w, dtype)
    toks = rng.integers(0, 60, 8300).tolist()
    eng = model.engine(1, 8300)
    rows = [0, 17, 5000, 8191, 8192, 8193, 8299]
    once = eng.forward(toks, want=rows)[0]
    eng.reset(0)
    parts, lo = [], 0
    for n in (3001, 1, 4100, 1198):
        here = [r - lo for r in rows if lo <= r < lo + n]
        parts.append(eng.forward(toks[lo:lo + n], want=here)[0])
        lo += n
    assert rel(once, np.concatenate(parts)) < TOL[dtype]
    batch = rng.integers(0, 60, (3, 3000)).astype(np.int32)
    eng3 = model.engine(3, 3000)
    both = eng3.forward(batch, want=[0, 2999, 3000 + 2730, 2 * 3000 + 2729, 2 * 3000 + 2999])[0]
    alone = []
    for i, r in ((0, [0, 2999]), (1, [2730]), (2, [2729, 2999])):
        eng.reset(0)
        alone.append(eng.forward(batch[i], want=r)[0])
    assert rel(both, np.concatenate(alone)) < TOL[dtype]
    assert gpu_dev.pipeline_status() == 0


def test_more_sequences_than_step_rows(gpu_dev):
    """Eighteen sequences: the linears of a step go to the GEMM, the mixers stay token by token."""
    from applegpu_runtime_b200.generate import greedy_generate
    cfg = CONFIGS["looped"]
    model = gpu_dev.load_gedenex(cfg, weights(cfg, 9), "float32")
    prompts = [np.random.default_rng(i).integers(0, cfg["vocab"], 3 + i).tolist() for i in range(18)]
    out = greedy_generate(model, prompts, 6)
    for i in (0, 7, 17):
        assert greedy_generate(model, [prompts[i]], 6)[0].tolist() == out[i]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation(gpu_dev, dtype):
    from applegpu_runtime_b200.generate import generate, greedy_generate
    cfg, g = CONFIGS["looped"], gpu_dev
    w = weights(cfg, 9)
    model = g.build_model(cfg, w, dtype)
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
            best = logits.max(-1)
            took = logits[np.arange(10), o[len(p):]]
            assert np.all(best - took < 0.1)
        assert generate(model, p, 10, temperature=0) == o
    square = greedy_generate(model, [prompts[0], prompts[2][:19]], 4)
    assert square.shape == (2, 23) and square[0].tolist() == out[0][:23]
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
    assert sorted(os.listdir(tmp_path)) == sorted(f"{i}.f32" for i in want)
    for i, ref in want.items():
        assert rel(np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]), ref) < TOL[dtype] * 3
