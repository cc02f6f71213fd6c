"""Model registry: config.json names the architecture, the registry knows how to load it.

`load_model(folder, dtype)` reads config.json and model.safetensors. Keys are the value of "architecture" (or the first of
"architectures", or "model_type"); a family registers a loader (config, {name: array}, dtype) -> model, where a model is what
`generate` and `greedy_generate` take.
"""
import json
import os

from .bert import BERT_BASE, load_bert_state_dict
from .checkpoint import read_safetensors
from .gedenex import ARCHITECTURE as _GEDENEX, load_gedenex
from .gpt2 import load_gpt2_state_dict
from .rurunex import ARCHITECTURE as _RURUNEX, load_rurunex

_LOADERS = {}


def register(name, loader):
    _LOADERS[name] = loader


def architecture_of(config):
    name = config.get("architecture") or (config.get("architectures") or [None])[0] or config.get("model_type")
    if name not in _LOADERS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(_LOADERS))}")
    return name


def build_model(config, weights, dtype="bfloat16"):
    return _LOADERS[architecture_of(config)](config, weights, dtype)


def load_model(folder, dtype="bfloat16"):
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    architecture_of(config)                       # before the weights are read
    return build_model(config, read_safetensors(os.path.join(folder, "model.safetensors")), dtype)


def _gpt2(config, weights, dtype):
    state = {n if n.startswith(("transformer.", "lm_head.")) else "transformer." + n: a for n, a in weights.items()}
    return load_gpt2_state_dict(state, {k: config[k] for k in ("n_layer", "n_head", "n_embd", "vocab_size", "n_positions")}, dtype=dtype)


_BERT_KEYS = {"n_layer": "num_hidden_layers", "n_head": "num_attention_heads", "n_embd": "hidden_size", "d_ff": "intermediate_size", "vocab_size": "vocab_size",
              "n_positions": "max_position_embeddings"}


def _bert(config, weights, dtype):
    cfg = {k: config[hf] if hf in config else config[k] for k, hf in _BERT_KEYS.items()}
    return load_bert_state_dict(weights, {**BERT_BASE, **cfg}, dtype=dtype)


for _n in ("gpt2", "GPT2LMHeadModel"):
    register(_n, _gpt2)
for _n in ("bert", "BertModel"):
    register(_n, _bert)
register(_GEDENEX, load_gedenex)
register(_RURUNEX, load_rurunex)
