"""Model folders through the registry: the families that were there before load and generate like models built by hand."""
import json

import numpy as np
import pytest

pytestmark = pytest.mark.gpu


def test_gpt2_folder(gpu_dev, tmp_path):
    from applegpu_runtime_b200.checkpoint import bf16_to_f32, f32_to_bf16, write_safetensors
    g = gpu_dev
    cfg = {"n_layer": 2, "n_head": 2, "n_embd": 128, "vocab_size": 96, "n_positions": 64}
    state = {n: t.to_numpy() for n, t in g.init_gpt2_weights(cfg, seed=4)["weights"].items()}
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["GPT2LMHeadModel"], "model_type": "gpt2", **cfg}))
    write_safetensors(str(tmp_path / "model.safetensors"), {n.removeprefix("transformer."): a for n, a in state.items()})
    by_hand = g.load_gpt2_state_dict({n: bf16_to_f32(f32_to_bf16(a)) for n, a in state.items()}, cfg, dtype="float32")
    model = g.load_model(str(tmp_path), "float32")
    ids = np.random.default_rng(0).integers(0, 96, (2, 9))
    assert np.array_equal(g.greedy_generate(model, ids, 8), g.greedy_generate(by_hand, ids, 8))
    assert np.array_equal(g.gpt2_forward(model, ids)[0].to_numpy(), g.gpt2_forward(by_hand, ids)[0].to_numpy())


def test_bert_folder(gpu_dev, tmp_path):
    from applegpu_runtime_b200.checkpoint import bf16_to_f32, f32_to_bf16, write_safetensors
    g = gpu_dev
    cfg = {**g.BERT_BASE, "n_layer": 1, "n_head": 2, "n_embd": 128, "d_ff": 256, "vocab_size": 80, "n_positions": 32}
    from applegpu_runtime_b200.modelbench import _bert_host_state
    state = {n: np.asarray(a, np.float32) for n, a in _bert_host_state(cfg, seed=4).items()}
    hf = {"num_hidden_layers": 1, "num_attention_heads": 2, "hidden_size": 128, "intermediate_size": 256, "vocab_size": 80, "max_position_embeddings": 32}
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "bert", **hf}))
    write_safetensors(str(tmp_path / "model.safetensors"), state)
    by_hand = g.load_bert_state_dict({n: bf16_to_f32(f32_to_bf16(a)) for n, a in state.items()}, cfg, dtype="float32")
    ids = np.random.default_rng(0).integers(0, 80, (2, 9))
    assert np.array_equal(g.bert_forward(g.load_model(str(tmp_path), "float32"), ids).to_numpy(), g.bert_forward(by_hand, ids).to_numpy())
