"""Plain float64 restatement of the Gedenex decoder, one function per mechanism (test oracle; numpy only).

Everything is written token by token or as whole matrices, the way the equations read; nothing is chunked, cached or
shared with the product code. Weights come as a {tensor name: array} dict, the configuration as the parsed config.json.
`State` keeps what a sequence carries from one call to the next, so the same functions also serve as a step-by-step
reference.
"""
import math

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, np.float64)))


def log_sigmoid(z):
    z = np.asarray(z, np.float64)
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps) * weight


def clamped_glu(gate, up, limit):
    """g sigmoid(1.702 g) (u + 1), g clipped from above, u on both sides."""
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def yarn_frequencies(rot):
    """(angle per position of every rotated pair, amplitude of cos and sin)."""
    n = rot["dims"]
    i = np.arange(n // 2, dtype=np.float64)
    freq = float(rot["base"]) ** (-2.0 * i / n)
    scaling = rot.get("scaling")
    if not scaling:
        return freq, 1.0

    def pair_turning(turns):      # the (fractional) pair whose wave turns this often within the original context
        return n * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))

    lo = max(math.floor(pair_turning(scaling["fast"])), 0)
    hi = min(math.ceil(pair_turning(scaling["slow"])), n - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq / scaling["factor"] * ramp + freq * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, positions, rot):
    """x [..., T, n]: pairs (2i, 2i + 1) of the first rot.dims entries turned by position * frequency."""
    freq, amp = yarn_frequencies(rot)
    ang = np.asarray(positions, np.float64)[:, None] * freq[None, :]
    c, s = np.cos(ang) * amp, np.sin(ang) * amp
    out = np.array(x, np.float64)
    n = rot["dims"]
    u, v = np.array(x[..., 0:n:2], np.float64), np.array(x[..., 1:n:2], np.float64)
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def mlstm_cell(q, k, v, log_i, log_f, S, n, m):
    """One token of one head: returns the read-out and the new (matrix memory, normaliser, running maximum)."""
    m_new = max(log_f + m, log_i)
    keep, write = math.exp(log_f + m - m_new), math.exp(log_i - m_new)
    S = keep * S + write * np.outer(k, v)
    n = keep * n + write * k
    o = (S.T @ q) / (max(abs(float(n @ q)), math.exp(-m_new)) + 1e-6)
    return o, S, n, m_new


def mlstm_sequence(q, k, v, log_i, log_f, state=None):
    """q, k [T, H, d], v [T, H, e], gates [T, H] -> [T, H, e] and the state after the last token."""
    T, H, d = q.shape
    e = v.shape[2]
    S, n, m = state if state is not None else (np.zeros((H, d, e)), np.zeros((H, d)), np.zeros(H))
    S, n, m = S.copy(), n.copy(), m.copy()
    out = np.zeros((T, H, e))
    for t in range(T):
        for h in range(H):
            out[t, h], S[h], n[h], m[h] = mlstm_cell(q[t, h], k[t, h], v[t, h], float(log_i[t, h]), float(log_f[t, h]), S[h], n[h], m[h])
    return out, (S, n, m)


def head_norm(o, eps):
    return o / np.sqrt(np.mean(np.square(o), axis=-1, keepdims=True) + eps)


def mlstm_mixer(h, w, prefix, mixer, eps, state=None):
    T = h.shape[0]
    H, d, e, cap = mixer["heads"], mixer["dim"], mixer["vdim"], float(mixer["gate_cap"])
    q = (h @ w[prefix + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[prefix + "k"].T).reshape(T, H, d)
    v = (h @ w[prefix + "v"].T).reshape(T, H, e)
    log_i = cap * np.tanh((h @ w[prefix + "i"].T + w[prefix + "i.b"]) / cap)
    log_f = log_sigmoid(cap * np.tanh((h @ w[prefix + "f"].T + w[prefix + "f.b"]) / cap))
    o, state = mlstm_sequence(q, k, v, log_i, log_f, state)
    y = head_norm(o, eps).reshape(T, H * e) * w[prefix + "norm"] * sigmoid(h @ w[prefix + "g"].T)
    return y @ w[prefix + "o"].T, state


def latent_attention_mixer(h, w, prefix, mixer, eps, state=None):
    """state: (latents [P, r], rotated keys [P, rot]) of the tokens before these."""
    T = h.shape[0]
    H, d, rd, e, r = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    past = 0 if state is None else state[0].shape[0]
    pos = np.arange(past, past + T)
    q = (h @ w[prefix + "q"].T).reshape(T, H, d + rd)
    q_plain, q_rot = q[..., :d], rotate_pairs(q[..., d:].transpose(1, 0, 2), pos, mixer["rot"]).transpose(1, 0, 2)
    down = h @ w[prefix + "dkv"].T
    c = rms_norm(down[:, :r], w[prefix + "dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, r:], pos, mixer["rot"])
    if past:
        c, k_rot = np.concatenate([state[0], c]), np.concatenate([state[1], k_rot])
    k_plain = (c @ w[prefix + "uk"].T).reshape(-1, H, d)
    v = (c @ w[prefix + "uv"].T).reshape(-1, H, e)
    out = np.zeros((T, H, e))
    for t in range(T):
        seen = past + t + 1
        for g in range(H):
            s = (k_plain[:seen, g] @ q_plain[t, g] + k_rot[:seen] @ q_rot[t, g]) * mixer["scale"]
            p = np.exp(s - s.max())
            out[t, g] = (p / p.sum()) @ v[:seen, g]
    return out.reshape(T, H * e) @ w[prefix + "o"].T, (c, k_rot)


MIXERS = {"mlstm": mlstm_mixer, "latent_attention": latent_attention_mixer}


def layer_runs(cfg):
    """The layer runs of one forward: (layer, pass of the loop or None, first layer of that pass?)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    runs = [(i, None, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None, False) for i in range(loop["stop"], n)]


def forward(cfg, weights, tokens, states=None, trace=None):
    """Logits [T, vocab] of the next T tokens of one sequence; `states` (one entry per layer run) is updated in place."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    runs = layer_runs(cfg)
    if states is None:
        states = [None] * len(runs)
    elif not states:
        states.extend([None] * len(runs))
    emb = w["embed"][np.asarray(tokens)]
    x = emb.copy()
    for r, (i, t, first) in enumerate(runs):
        if first:
            if t > 0:
                x = x + emb
            x = x + w["loop.step"][t]
        layer = cfg["layers"][i]
        p = f"l{i}."
        y, states[r] = MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps, states[r])
        if layer.get("mlp"):
            h = rms_norm(x, w[p + "norm2"], eps)
            y = y + clamped_glu(h @ w[p + "mlp.gate"].T, h @ w[p + "mlp.up"].T, layer["mlp"]["limit"]) @ w[p + "mlp.down"].T
        x = x + y
        if trace is not None:
            trace.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
