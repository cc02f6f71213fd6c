"""Gedenex: mLSTM and latent-attention layers, each beside a clamped gated feed-forward, part of them looped.

config.json: "layers" [{"type", "mixer", "mlp"}], "loop" {"start", "stop", "times"}, "norm" {"eps"}, "vocab", "width".
Tensors: embed, head, final.norm, loop.step, and per layer l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.{gate,up,down}; linear
weights are [out, in].
"""
import numpy as np

from .seqmodel import Layer, SequenceModel, Tensors, interleaved, rotary_of, rows, side_by_side

ARCHITECTURE = "Gedenex"


def _mlstm(t, p, m, width):
    H, d, e = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    layer = Layer("mlstm", heads=H, dim=d, vdim=e, gate_cap=float(m["gate_cap"]))
    layer.w_in = rows(t.get(p + "q", H * d, width), t.get(p + "k", H * d, width), t.get(p + "v", H * e, width), t.get(p + "g", H * e, width))
    layer.own = [rows(t.get(p + "i", H, width), t.get(p + "f", H, width)), np.concatenate([t.get(p + "i.b", H), t.get(p + "f.b", H)]), t.get(p + "norm", H * e)]
    return layer


def _latent_attention(t, p, m, width):
    H, d, rd, e, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    layer = Layer("latent_attention", heads=H, dim=d, vdim=e, rot_dim=rd, kv_rank=r, score_scale=float(m["scale"]))
    layer.rotary = rotary_of(m.get("rot"))
    if layer.rotary and (layer.rotary.dims > rd or layer.rotary.dims % 2):
        raise ValueError(f"{p}: {layer.rotary.dims} rotated dimensions of {rd}")
    layer.w_in = rows(t.get(p + "q", H * (d + rd), width), t.get(p + "dkv", r + rd, width))
    layer.own = [t.get(p + "dkv.norm", r), rows(t.get(p + "uk", H * d, r), t.get(p + "uv", H * e, r), pad_rows=True), None]
    return layer


_MIXERS = {"mlstm": _mlstm, "latent_attention": _latent_attention}


def load_gedenex(config, weights, dtype="bfloat16"):
    """A SequenceModel from the parsed config.json and {tensor name: array}."""
    width, vocab, t = int(config["width"]), int(config["vocab"]), Tensors(weights)
    layers = []
    for i, c in enumerate(config["layers"]):
        if c["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {c['type']}")
        p = f"l{i}."
        layer = _MIXERS[c["type"]](t, p + "mix.", c["mixer"], width)
        out = t.get(p + "mix.o", width, layer.heads * layer.vdim)
        layer.norm1 = t.get(p + "norm1", width)
        mlp, down = c.get("mlp"), None
        if mlp:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']}")
            layer.ff, layer.ff_limit = int(mlp["ff"]), float(mlp["limit"])
            layer.norm2 = t.get(p + "norm2", width)
            layer.w_ff = interleaved(t.get(p + "mlp.gate", layer.ff, width), t.get(p + "mlp.up", layer.ff, width))
            down = t.get(p + "mlp.down", width, layer.ff)
        layer.w_out = side_by_side(out, down)
        layers.append(layer)
    loop = config.get("loop")
    if loop and int(loop["times"]) > 0 and int(loop["stop"]) > int(loop["start"]):
        loop = (int(loop["start"]), int(loop["stop"]), t.get("loop.step", int(loop["times"]), width))
    else:
        loop = None
    return SequenceModel(vocab, width, config["norm"]["eps"], layers, t.get("embed", vocab, width), t.get("head", vocab, width), t.get("final.norm", width), loop=loop,
                         dtype=dtype, config=dict(config))


def init_gedenex_weights(config, seed=0, std=0.02):
    """Random weights for a configuration, {tensor name: float32 array}: N(0, std) matrices, unit norms, zero biases."""
    rng = np.random.default_rng(seed)
    W, V, w = int(config["width"]), int(config["vocab"]), {}

    def mat(name, *shape):
        w[name] = (rng.standard_normal(shape, dtype=np.float32) * np.float32(std)).astype(np.float32)

    def ones(name, n):
        w[name] = np.ones(n, np.float32)

    mat("embed", V, W)
    mat("head", V, W)
    ones("final.norm", W)
    if config.get("loop"):
        mat("loop.step", int(config["loop"]["times"]), W)
    for i, c in enumerate(config["layers"]):
        m, p = c["mixer"], f"l{i}."
        H, d, e = m["heads"], m["dim"], m["vdim"]
        ones(p + "norm1", W)
        if c["type"] == "mlstm":
            for n, k in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e), ("i", H), ("f", H)):
                mat(p + "mix." + n, k, W)
            w[p + "mix.i.b"], w[p + "mix.f.b"] = np.zeros(H, np.float32), np.full(H, 3.0, np.float32)
            ones(p + "mix.norm", H * e)
        else:
            mat(p + "mix.q", H * (d + m["rot_dim"]), W)
            mat(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], W)
            ones(p + "mix.dkv.norm", m["kv_rank"])
            mat(p + "mix.uk", H * d, m["kv_rank"])
            mat(p + "mix.uv", H * e, m["kv_rank"])
        mat(p + "mix.o", W, H * e)
        if c.get("mlp"):
            ones(p + "norm2", W)
            mat(p + "mlp.gate", c["mlp"]["ff"], W)
            mat(p + "mlp.up", c["mlp"]["ff"], W)
            mat(p + "mlp.down", W, c["mlp"]["ff"])
    return w
