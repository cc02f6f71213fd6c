"""Sequence models: decoder-only models made of layers with per-sequence memory (recurrent states, key caches).

A `SequenceModel` holds uploaded weights and the list of layers; `engine(slots, max_len)` gives them memory for that many
sequences and runs prompt portions and generated tokens (csrc/core/seqmodel.cc). A model family is a module that turns
its configuration and tensor names into one (`gedenex.py`, `rurunex.py`); it packs the weights with the helpers here and adds nothing
to the run time.
"""
import ctypes
from dataclasses import dataclass, field

import numpy as np

from . import _lib
from . import api as gpu
from .rotary import rotary_table

MIXERS = {"mlstm": 1, "latent_attention": 2, "key_decay": 3, "grouped_attention": 4}
FORMS = {"parallel": 0, "sequential": 1}
GLUS = {"clamped": 0, "silu": 1}
DELTA, UNIT, SOFTPLUS, GATE_SILU = 1, 2, 4, 8          # key_decay options


def pad8(n):
    return (n + 7) // 8 * 8


class _ModelDesc(ctypes.Structure):
    _fields_ = [(n, ctypes.c_int32) for n in ("vocab", "width", "n_layers", "loop_start", "loop_stop", "loop_times", "form")] + [("eps", ctypes.c_float), ("embed_scale", ctypes.c_float)]


class _LayerDesc(ctypes.Structure):
    _fields_ = ([(n, ctypes.c_int32) for n in ("mixer", "heads", "dim", "vdim", "rot_dim", "rot_pairs", "kv_rank", "ff", "kv_heads", "window", "kv_from", "taps",
                                                 "a_rank", "g_rank", "flags", "glu")]
                + [(n, ctypes.c_float) for n in ("gate_cap", "score_scale", "ff_limit", "softcap", "tau")])


@dataclass
class Rotary:
    dims: int
    base: float
    scaling: dict = None       # factor, original, fast, slow


@dataclass
class Layer:
    """One layer: the mixer kind with its constants, the feed-forward, and the weights in the engine's order (None where a
    layer has none; matrices as padded by `rows`, vectors as float32)."""
    mixer: str
    heads: int
    dim: int
    vdim: int
    rot_dim: int = 0
    kv_rank: int = 0
    gate_cap: float = 0.0
    score_scale: float = 0.0
    rotary: Rotary = None
    kv_heads: int = 0          # grouped_attention, key_decay
    window: int = 0            # keys a token sees, 0: all
    kv_from: int = -1          # layer whose keys and values are used, -1: its own
    softcap: float = 0.0
    taps: int = 0
    a_rank: int = 0
    g_rank: int = 0
    flags: int = 0
    tau: float = 1.0
    ff: int = 0
    glu: str = "clamped"
    ff_limit: float = 0.0
    norm1: np.ndarray = None
    norm2: np.ndarray = None
    w_in: np.ndarray = None
    w_out: np.ndarray = None
    w_ff: np.ndarray = None
    post1: np.ndarray = None   # sequential layers: norms behind the sublayers, feed-forward output
    post2: np.ndarray = None
    w_down: np.ndarray = None
    own: list = field(default_factory=lambda: [None] * 7)

    def weights(self):
        own = self.own + [None] * (7 - len(self.own))
        return [self.norm1, self.norm2, self.w_in, self.w_out, self.w_ff, *own[:3], self.post1, self.post2, self.w_down, *own[3:]]


LAYER_WEIGHTS, ROTATION = 15, 7        # records per layer, place of the rotation table among them


class Tensors:
    """Looks weights up by name and checks their shapes."""

    def __init__(self, weights):
        self._w = weights

    def get(self, name, *shape):
        if name not in self._w:
            raise ValueError(f"missing tensor {name}")
        a = np.asarray(self._w[name], np.float32)
        if a.shape != tuple(shape):
            raise ValueError(f"tensor {name} has shape {list(a.shape)}, the configuration asks for {list(shape)}")
        return a

    def rank(self, name):
        """Number of rows of a matrix whose size only its shape tells."""
        if name not in self._w:
            raise ValueError(f"missing tensor {name}")
        return int(np.shape(self._w[name])[0])


def rotary_of(rot):
    """The `Rotary` of a configuration's "rot" entry (dims, base, optional scaling), None without one."""
    if not rot or not int(rot["dims"]):
        return None
    scaling = rot.get("scaling")
    return Rotary(int(rot["dims"]), float(rot["base"]), None if not scaling else {k: float(scaling[k]) for k in ("factor", "original", "fast", "slow")})


def rows(*parts, pad_rows=False):
    """[out, in] matrices stacked along `out`, the length of a row padded with zeros to a multiple of 8; `pad_rows` also pads
    every part's number of rows."""
    k = parts[0].shape[1]
    out = []
    for p in parts:
        if p.ndim != 2 or p.shape[1] != k:
            raise ValueError(f"matrices of different input sizes stacked: {[q.shape for q in parts]}")
        n = pad8(p.shape[0]) if pad_rows else p.shape[0]
        a = np.zeros((n, pad8(k)), np.float32)
        a[:p.shape[0], :k] = p
        out.append(a)
    return np.concatenate(out, axis=0)


def interleaved(gate, up, block=16):
    """Gate and up rows in blocks of 16 gates and the 16 rows they gate, padded with zero rows to whole blocks."""
    n = (gate.shape[0] + block - 1) // block
    a = np.zeros((n, 2, block, gate.shape[1]), np.float32)
    for i, p in enumerate((gate, up)):
        q = np.zeros((n * block, gate.shape[1]), np.float32)
        q[:p.shape[0]] = p
        a[:, i] = q.reshape(n, block, -1)
    return rows(a.reshape(2 * n * block, -1))


def side_by_side(first, second):
    """Two [out, in] matrices with their inputs one after the other, the first one's padded to a multiple of 8."""
    if second is None:
        return rows(first)
    a = np.zeros((first.shape[0], pad8(pad8(first.shape[1]) + second.shape[1])), np.float32)
    a[:, :first.shape[1]] = first
    a[:, pad8(first.shape[1]):pad8(first.shape[1]) + second.shape[1]] = second
    return a


class SequenceModel:
    def __init__(self, vocab, width, eps, layers, embed, head, final_norm, loop=None, dtype="bfloat16", config=None, form="parallel", embed_scale=1.0):
        """`loop`: (start, stop, step vectors [times, width]) or None; `form`: how a layer's sublayers meet the stream
        (csrc/core/seqmodel.cc). Arrays are float32; matrices are stored as `dtype`."""
        if dtype not in ("float32", "bfloat16", "float16"):
            raise ValueError(f"sequence models run in float32, bfloat16 or float16, not {dtype}")
        self.vocab, self.width, self.eps, self.dtype, self.layers, self.config = int(vocab), int(width), float(eps), dtype, layers, config
        self.form, self.embed_scale = form, float(embed_scale)
        self.loop = None if loop is None else (int(loop[0]), int(loop[1]), int(loop[2].shape[0]))
        self._weights = [self._matrix(np.asarray(embed, np.float32)), self._matrix(rows(head)), self._vector(final_norm), self._vector(loop[2]) if loop else None]
        for l in layers:
            self._weights += [a if a is None else (self._matrix(a) if a.ndim == 2 else self._vector(a)) for a in l.weights()]
            l.norm1 = l.norm2 = l.w_in = l.w_out = l.w_ff = l.post1 = l.post2 = l.w_down = None      # uploaded
            l.own = []

    @staticmethod
    def _vector(a):
        return None if a is None else gpu.from_numpy(np.ascontiguousarray(a, np.float32))

    def _matrix(self, a):
        if a is None:
            return None
        t = gpu.from_numpy(np.ascontiguousarray(a, np.float32))
        if self.dtype != "float32":
            t = gpu.cast(t, self.dtype)
            t.eval()
        return t

    def engine(self, slots=1, max_len=2048):
        return SequenceEngine(self, slots, max_len)


class SequenceEngine:
    """Memory for `slots` sequences of at most `max_len` tokens and the step functions over them. Slots are handed out by
    `acquire` and given back by `release`, which empties them."""

    def __init__(self, model, slots, max_len):
        self._lib = _lib.load()
        self.model, self.slots, self.max_len = model, int(slots), int(max_len)
        tables, w = {}, list(model._weights)
        desc = _ModelDesc(model.vocab, model.width, len(model.layers), *(model.loop or (0, 0, 0)), FORMS[model.form], model.eps, model.embed_scale)
        arr = (_LayerDesc * len(model.layers))()
        for i, l in enumerate(model.layers):
            pairs = 0
            if l.rotary is not None and l.rotary.dims:
                pairs = l.rotary.dims // 2
                key = (l.rotary.dims, l.rotary.base, tuple(sorted((l.rotary.scaling or {}).items())))
                if key not in tables:
                    tables[key] = gpu.from_numpy(rotary_table(self.max_len, l.rotary.dims, l.rotary.base, l.rotary.scaling))
                w[4 + LAYER_WEIGHTS * i + ROTATION] = tables[key]
            arr[i] = _LayerDesc(MIXERS[l.mixer], l.heads, l.dim, l.vdim, l.rot_dim, pairs, l.kv_rank, l.ff, l.kv_heads, l.window, l.kv_from, l.taps,
                                l.a_rank, l.g_rank, l.flags, GLUS[l.glu], l.gate_cap, l.score_scale, l.ff_limit, l.softcap, l.tau)
        self._keep = w
        ids = (ctypes.c_uint64 * len(w))(*[0 if t is None else t.id for t in w])
        self.handle = int(self._lib.applegpu_seq_create(ctypes.byref(desc), arr, ids, len(w), self.slots, self.max_len))
        if not self.handle:
            raise ValueError(gpu._err())
        self._free = list(range(self.slots))

    # slots
    def acquire(self):
        if not self._free:
            raise RuntimeError(f"all {self.slots} sequence slots are taken")
        return self._free.pop(0)

    def release(self, slot):
        self.reset(slot)
        self._free.append(slot)
        self._free.sort()

    def reset(self, slot=0, n=1):
        self._check(self._lib.applegpu_seq_reset(self.handle, slot, n))

    def length(self, slot):
        return int(self._lib.applegpu_seq_length(self.handle, slot))

    # steps
    def forward(self, tokens, slot=0, want=None, logits=True, pick=False, layers=False):
        """The next tokens of one sequence ([T]) or of n sequences in consecutive slots ([n, T]). `want`: the rows (s * T + t)
        whose results are asked for, by default the last one of every sequence. Returns (logits [n_want, vocab] or None,
        greedy picks [n_want] or None), with `layers` also the residual stream after every layer run [runs, n * T, width]."""
        tok = np.ascontiguousarray(tokens, np.int32)
        if tok.ndim == 1:
            tok = tok[None]
        n, T = tok.shape
        want = np.ascontiguousarray([s * T + T - 1 for s in range(n)] if want is None else want, np.int32)
        out = np.empty((want.size, self.model.vocab), np.float32) if logits else None
        picked = np.empty(want.size, np.int32) if pick else None
        runs = int(self._lib.applegpu_seq_info(self.handle, 2))
        stream = np.empty((runs, n * T, self.model.width), np.float32) if layers else None

        def ptr(a):
            return None if a is None or a.size == 0 else a.ctypes.data_as(ctypes.c_void_p)
        self._check(self._lib.applegpu_seq_forward(self.handle, slot, n, ptr(tok), T, ptr(want), want.size, ptr(out), ptr(picked), ptr(stream)))
        return (out, picked, stream) if layers else (out, picked)

    def decode(self, n_steps, slot=0, n=1, use_graph=True):
        """n_steps greedy tokens for n sequences, continuing from the last `forward(pick=True)`: int32 [n_steps, n]."""
        out = np.empty((int(n_steps), n), np.int32)
        if n_steps > 0:
            self._check(self._lib.applegpu_seq_decode(self.handle, slot, n, int(n_steps), out.ctypes.data_as(ctypes.c_void_p), bool(use_graph)))
        return out

    @property
    def launches_per_step(self):
        return int(self._lib.applegpu_seq_info(self.handle, 0))

    @property
    def uses_graph(self):
        return int(self._lib.applegpu_seq_info(self.handle, 1)) == 1

    def _check(self, rc):
        if rc != 0:
            raise ValueError(gpu._err())

    def close(self):
        if self.handle:
            self._lib.applegpu_seq_destroy(self.handle)
            self.handle = 0

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass


def greedy_generate(model, prompts, max_tokens, use_graph=True, engine=None):
    """Greedy continuation of prompts of any lengths: a list of token lists, each prompt + generated. Prompts of one length
    run as one portion, others one by one; the generated tokens of all sequences go through one step at a time."""
    prompts = [np.asarray(p, np.int32).reshape(-1) for p in prompts]
    if not prompts or min(p.size for p in prompts) < 1:
        raise ValueError("every prompt needs at least one token")
    if max_tokens <= 0:
        return [p.tolist() for p in prompts]
    n = len(prompts)
    eng = engine or model.engine(slots=n, max_len=max(p.size for p in prompts) + max_tokens)
    try:
        eng.reset(0, n)
        if len({p.size for p in prompts}) == 1:
            first = eng.forward(np.stack(prompts), logits=False, pick=True)[1]
        else:
            first = np.concatenate([eng.forward(p, slot=i, logits=False, pick=True)[1] for i, p in enumerate(prompts)])
        # the picks of separate portions are handed to the joint step as its tokens
        new = [first]
        if max_tokens > 1:
            new.append(eng.forward(first[:, None], logits=False, pick=True)[1])
        if max_tokens > 2:
            new.extend(eng.decode(max_tokens - 2, 0, n, use_graph))
        stats = {"launches_per_step": eng.launches_per_step, "graph": eng.uses_graph}
    finally:
        if engine is None:
            eng.close()
    model.last_decode_stats = stats
    new = np.stack(new, axis=1)
    return [p.tolist() + new[i].tolist() for i, p in enumerate(prompts)]


def sample_generate(model, prompt, max_tokens, pick_token, engine=None):
    """Generation with a host-side choice: `pick_token` turns a row of logits into a token id."""
    ids = list(prompt)
    eng = engine or model.engine(slots=1, max_len=len(ids) + max_tokens)
    try:
        eng.reset(0, 1)
        nxt = ids
        for _ in range(max_tokens):
            logits, _ = eng.forward(nxt)
            nxt = [int(pick_token(logits[0]))]
            ids += nxt
    finally:
        if engine is None:
            eng.close()
    return ids
