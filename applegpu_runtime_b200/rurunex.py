"""Rurunex: sequential layers with norms on both sides of each sublayer; gated linear attention, the channel-wise gated delta
rule and windowed grouped attention (which may use an earlier layer's keys and values), silu-gated feed-forwards.

config.json: "embedding" {"scale"}, "layers" [{"type", "mixer", "mlp"}], "norm" {"eps"}, "logit_scale", "vocab", "width".
Tensors: embed, head, final.norm, and per layer l<i>.norm1, norm1b, norm2, norm2b, l<i>.mix.*, l<i>.mlp.{gate,up,down}; linear
weights are [out, in]. The norms around sublayers and the final one store their weight's difference from one.
"""
import numpy as np

from .seqmodel import DELTA, GATE_SILU, SOFTPLUS, UNIT, Layer, SequenceModel, Tensors, interleaved, rotary_of, rows

ARCHITECTURE = "Rurunex"


def _gla(t, p, m, width):
    H, d, e, r = int(m["heads"]), int(m["dim"]), int(m["vdim"]), t.rank(p + "a1")
    layer = Layer("key_decay", heads=H, dim=d, vdim=e, kv_heads=H, a_rank=r, tau=float(m["tau"]), flags=GATE_SILU)
    layer.w_in = rows(t.get(p + "q", H * d, width), t.get(p + "k", H * d, width), t.get(p + "v", H * e, width), t.get(p + "a1", r, width), t.get(p + "g", H * e, width), pad_rows=True)
    layer.own = [None, rows(t.get(p + "a2", H * d, r)), t.get(p + "a2.b", H * d), t.get(p + "norm", e)]
    return layer


def _channel_delta(t, p, m, width):
    H, G, d, e, n = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"])
    r, s = t.rank(p + "a1"), t.rank(p + "g1")
    if H % G:
        raise ValueError(f"{p}: {H} heads over {G} query / key heads")
    layer = Layer("key_decay", heads=H, dim=d, vdim=e, kv_heads=G, a_rank=r, g_rank=s, taps=n, flags=DELTA | UNIT | SOFTPLUS)
    layer.w_in = rows(t.get(p + "q", G * d, width), t.get(p + "k", G * d, width), t.get(p + "v", H * e, width), t.get(p + "a1", r, width), t.get(p + "g1", s, width), pad_rows=True)
    conv = np.concatenate([t.get(p + "q.conv", G * d, n), t.get(p + "k.conv", G * d, n), t.get(p + "v.conv", H * e, n)])
    layer.own = [rows(t.get(p + "b", H, width)), rows(t.get(p + "a2", H * d, r)), t.get(p + "dt_bias", H * d), t.get(p + "norm", e), rows(t.get(p + "g2", H * e, s)),
                 np.exp(t.get(p + "A_log", H)), conv.reshape(-1)]
    return layer


def _attention(t, p, m, width):
    H, G, d, e = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    if H % G:
        raise ValueError(f"{p}: {H} heads over {G} key heads")
    mask, source = m.get("mask"), m.get("kv_from")
    layer = Layer("grouped_attention", heads=H, dim=d, vdim=e, kv_heads=G, window=int(mask["size"]) if mask else 0, kv_from=-1 if source is None else int(source),
                  softcap=float(m.get("softcap") or 0.0), score_scale=float(m["scale"]), rotary=rotary_of(m.get("rot")))
    if layer.rotary and (layer.rotary.dims > d or layer.rotary.dims % 2):
        raise ValueError(f"{p}: {layer.rotary.dims} rotated dimensions of {d}")
    parts = [t.get(p + "q", H * d, width)]
    layer.own = [t.get(p + "q.norm", d), None, None]
    if source is None:
        parts += [t.get(p + "k", G * d, width), t.get(p + "v", G * e, width)]
        layer.own[1] = t.get(p + "k.norm", d)
    layer.w_in = rows(*parts, pad_rows=True)
    return layer


_MIXERS = {"gla": _gla, "channel_delta": _channel_delta, "attention": _attention}


def load_rurunex(config, weights, dtype="bfloat16"):
    """A SequenceModel from the parsed config.json and {tensor name: array}."""
    width, vocab, t = int(config["width"]), int(config["vocab"]), Tensors(weights)
    layers = []
    for i, c in enumerate(config["layers"]):
        if c["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {c['type']}")
        p = f"l{i}."
        layer = _MIXERS[c["type"]](t, p + "mix.", c["mixer"], width)
        layer.w_out = rows(t.get(p + "mix.o", width, layer.heads * layer.vdim))
        layer.norm1, layer.post1 = 1.0 + t.get(p + "norm1", width), 1.0 + t.get(p + "norm1b", width)
        mlp = c.get("mlp")
        if mlp:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']}")
            layer.ff, layer.glu = int(mlp["ff"]), "silu"
            layer.norm2, layer.post2 = 1.0 + t.get(p + "norm2", width), 1.0 + t.get(p + "norm2b", width)
            layer.w_ff = interleaved(t.get(p + "mlp.gate", layer.ff, width), t.get(p + "mlp.up", layer.ff, width))
            layer.w_down = rows(t.get(p + "mlp.down", width, layer.ff))
        layers.append(layer)
    # the factor on the logits rides in the weight of the norm ahead of the head
    final = (1.0 + t.get("final.norm", width)) * np.float32(config["logit_scale"])
    return SequenceModel(vocab, width, config["norm"]["eps"], layers, t.get("embed", vocab, width), t.get("head", vocab, width), final, dtype=dtype, config=dict(config),
                         form="sequential", embed_scale=config["embedding"]["scale"])


def init_rurunex_weights(config, seed=0, std=0.02, ranks=None):
    """Random weights for a configuration, {tensor name: float32 array}: N(0, std) matrices, unit norms, decays that keep most of a
    state; `ranks`: inner size of the two-step projections per mixer type."""
    rng = np.random.default_rng(seed)
    ranks = {"gla": 16, "channel_delta": 16, **(ranks or {})}
    W, V, w = int(config["width"]), int(config["vocab"]), {}

    def mat(name, *shape):
        w[name] = (rng.standard_normal(shape, dtype=np.float32) * np.float32(std)).astype(np.float32)

    mat("embed", V, W)
    mat("head", V, W)
    w["final.norm"] = np.zeros(W, np.float32)
    for i, c in enumerate(config["layers"]):
        m, p = c["mixer"], f"l{i}."
        x, H, d, e = p + "mix.", m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"] = np.zeros(W, np.float32), np.zeros(W, np.float32)
        if c["type"] == "attention":
            mat(x + "q", H * d, W)
            w[x + "q.norm"] = np.ones(d, np.float32)
            if m.get("kv_from") is None:
                mat(x + "k", m["kv_heads"] * d, W)
                mat(x + "v", m["kv_heads"] * e, W)
                w[x + "k.norm"] = np.ones(d, np.float32)
        else:
            G, r = m.get("kv_heads", H), ranks[c["type"]]
            for n, k in (("q", G * d), ("k", G * d), ("v", H * e), ("a1", r)):
                mat(x + n, k, W)
            mat(x + "a2", H * d, r)
            w[x + "norm"] = np.ones(e, np.float32)
            if c["type"] == "gla":
                mat(x + "g", H * e, W)
                w[x + "a2.b"] = np.zeros(H * d, np.float32)
            else:
                for n, k in (("q", G * d), ("k", G * d), ("v", H * e)):
                    w[x + n + ".conv"] = (rng.standard_normal((k, m["conv"])) * 0.5).astype(np.float32)
                mat(x + "b", H, W)
                mat(x + "g1", r, W)
                mat(x + "g2", H * e, r)
                w[x + "A_log"] = np.log(rng.uniform(0.5, 4.0, H)).astype(np.float32)
                w[x + "dt_bias"] = rng.uniform(-5.0, -2.0, H * d).astype(np.float32)
        mat(x + "o", W, H * e)
        if c.get("mlp"):
            w[p + "norm2"], w[p + "norm2b"] = np.zeros(W, np.float32), np.zeros(W, np.float32)
            mat(p + "mlp.gate", c["mlp"]["ff"], W)
            mat(p + "mlp.up", c["mlp"]["ff"], W)
            mat(p + "mlp.down", W, c["mlp"]["ff"])
    return w
