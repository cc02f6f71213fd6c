"""Plain float64 restatement of the Rurunex decoder, one function per mechanism (test oracle; numpy only).

Recurrences go token by token, attention row by row; nothing is chunked or shared with the product code. Weights come as a
{tensor name: array} dict, the configuration as the parsed config.json. A layer's state is whatever its mixer returns; a list
of them carries a sequence from one call of `forward` to the next.
"""
import numpy as np

from .gedenex_ref import log_sigmoid, rms_norm, sigmoid, yarn_frequencies


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its difference from one."""
    return rms_norm(x, 1.0 + w, eps)


def unit(x):
    return x / np.sqrt(np.sum(np.square(x), axis=-1, keepdims=True) + 1e-6)


def rotate_halves(x, positions, rot):
    """x [T, heads, dim]: entries i and i + dims / 2 of the first rot.dims turned as a pair."""
    freq, amp = yarn_frequencies(rot)
    ang = (np.asarray(positions, np.float64)[:, None] * freq[None, :])[:, None, :]
    c, s = np.cos(ang) * amp, np.sin(ang) * amp
    n = rot["dims"]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., n:]], axis=-1)


def causal_conv(x, taps, before):
    """x [T, channels], taps [channels, n] (the last one meets the current token), before: the n - 1 inputs ahead of x."""
    n = taps.shape[1]
    ext = np.concatenate([before, x])
    y = sum(ext[i:i + x.shape[0]] * taps[:, i] for i in range(n))
    return y, ext[ext.shape[0] - (n - 1):]


def gla_recurrence(q, k, v, alpha, S):
    """q, k, alpha [T, H, d], v [T, H, e], S [H, d, e] -> outputs [T, H, e] and the last state."""
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out, S


def delta_recurrence(q, k, v, g, beta, S):
    """As above with the delta rule: what S already returns for k is taken off v, the rest is written with strength beta."""
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out, S


def gla_mixer(h, w, p, m, eps, state, _):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, e)
    z = h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = np.exp(log_sigmoid(z) / m["tau"]).reshape(T, H, d)
    o, S = gla_recurrence(q, k, v, alpha, np.zeros((H, d, e)) if state is None else state)
    y = rms_norm(o, w[p + "norm"], eps).reshape(T, H * e) * silu(h @ w[p + "g"].T)
    return y @ w[p + "o"].T, S


def delta_mixer(h, w, p, m, eps, state, _):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    parts, tails = [], []
    for i, n in enumerate("qkv"):
        x = h @ w[p + n].T
        taps = w[p + n + ".conv"]
        before = np.zeros((taps.shape[1] - 1, x.shape[1])) if state is None else state[1][i]
        y, tail = causal_conv(x, taps, before)
        parts.append(silu(y))
        tails.append(tail)
    q = np.repeat(unit(parts[0].reshape(T, G, d)) * d ** -0.5, H // G, axis=1)
    k = np.repeat(unit(parts[1].reshape(T, G, d)), H // G, axis=1)
    v = parts[2].reshape(T, H, e)
    beta = sigmoid(h @ w[p + "b"].T)
    step = softplus(h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, d)
    g = np.exp(-np.exp(w[p + "A_log"])[:, None] * step)
    o, S = delta_recurrence(q, k, v, g, beta, np.zeros((H, d, e)) if state is None else state[0])
    gate = sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T)
    y = rms_norm(o, w[p + "norm"], eps).reshape(T, H * e) * gate
    return y @ w[p + "o"].T, (S, tails)


def attention_rows(q, k, v, past, scale, softcap, window):
    """q [T, H, d] of the tokens past .. past + T over k, v [past + T, G, ..] -> [T, H, e]."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        i = past + t
        lo = max(0, i - window + 1) if window else 0
        for h in range(H):
            s = k[lo:i + 1, h // group] @ q[t, h] * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            a = np.exp(s - s.max())
            out[t, h] = (a / a.sum()) @ v[lo:i + 1, h // group]
    return out


def attention_mixer(h, w, p, m, eps, state, source):
    """state: (keys, values) of the tokens so far; `source`: those of the layer whose keys this one uses, current tokens included."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    if source is None:
        past = 0 if state is None else state[0].shape[0]
    else:
        past = source[0].shape[0] - T
    pos = np.arange(past, past + T)
    q = rotate_halves(rms_norm((h @ w[p + "q"].T).reshape(T, H, d), w[p + "q.norm"], eps), pos, m["rot"])
    if source is None:
        k = rotate_halves(rms_norm((h @ w[p + "k"].T).reshape(T, G, d), w[p + "k.norm"], eps), pos, m["rot"])
        v = (h @ w[p + "v"].T).reshape(T, G, e)
        if past:
            k, v = np.concatenate([state[0], k]), np.concatenate([state[1], v])
        source = (k, v)
    mask = m.get("mask")
    o = attention_rows(q, source[0], source[1], past, m["scale"], m.get("softcap"), mask["size"] if mask else None)
    return o.reshape(T, H * e) @ w[p + "o"].T, source


MIXERS = {"gla": gla_mixer, "channel_delta": delta_mixer, "attention": attention_mixer}


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, weights, tokens, states=None, trace=None):
    """Logits [T, vocab] of the next T tokens of one sequence; `states` (one entry per layer) is updated in place."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, layers = cfg["norm"]["eps"], cfg["layers"]
    if states is None:
        states = []
    if not states:
        states.extend([None] * len(layers))
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(layers):
        p, m = f"l{i}.", layer["mixer"]
        source = None if m.get("kv_from") is None else states[m["kv_from"]]
        y, states[i] = MIXERS[layer["type"]](centred_norm(x, w[p + "norm1"], eps), w, p + "mix.", m, eps, states[i], source)
        x = x + centred_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
            x = x + centred_norm(y, w[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x.copy())
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
