"""Throughput of the sequence-model designs at equal size, and what their kernels reach of the roofline.

A size is a width; the mixers and feed-forwards take sizes a trained model of that width would have, weights are random
(N(0, 0.02)), token ids uniform. The GPT-2 of equal size has the same width, one layer per layer run, heads of 64 and a
feed-forward of four widths. Prefill: prompts of 1024 tokens, 8 at a time. Decode: greedy steps behind 1024-token prompts
through the captured step. Times are CUDA events on the runtime stream after warm-up; the weights and activations of a
forward exceed the L2.
"""
import time

import numpy as np

from . import _lib
from . import api as gpu
from .gedenex import init_gedenex_weights, load_gedenex
from .generate import Gpt2Decoder
from .gpt2 import gpt2_forward, init_gpt2_weights
from .rurunex import init_rurunex_weights, load_rurunex

SIZES = {1024: dict(heads=4, latent_heads=8, kv_rank=256, ff=2816), 2048: dict(heads=8, latent_heads=16, kv_rank=512, ff=5632)}
RURUNEX_SIZES = {1024: dict(gla=4, delta=8, heads=8, kv_heads=2, ff=2816), 2048: dict(gla=8, delta=16, heads=16, kv_heads=4, ff=5632)}
BYTES = ("rms_rows", "linear_gates", "clamped_glu", "mlstm_prefill", "mlstm_step", "latent_append", "latent_decode", "gla_prefill", "delta_prefill", "gla_step", "delta_step",
         "grouped_append", "grouped_decode", "skinny_in", "skinny_ff", "skinny_out", "skinny_head")


def config_of(width, vocab=32768):
    s = SIZES[width]
    mlp = {"kind": "dense", "ff": s["ff"], "limit": 7.0}
    ml = {"type": "mlstm", "mixer": {"heads": s["heads"], "dim": 128, "vdim": width // s["heads"], "gate_cap": 15.0}, "mlp": mlp}
    la = {"type": "latent_attention", "mlp": mlp,
          "mixer": {"heads": s["latent_heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": s["kv_rank"], "scale": 192 ** -0.5,
                    "rot": {"dims": 64, "base": 10000.0, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    return {"architecture": "Gedenex", "layers": [ml, ml, la, ml, ml, la], "loop": {"start": 0, "stop": 3, "times": 2}, "norm": {"eps": 1e-5}, "vocab": vocab, "width": width}


def rurunex_config_of(width, vocab=32768):
    """Nine layers like the nine layer runs above: matrix states of the same sizes, attention behind a window of 512 tokens."""
    s = RURUNEX_SIZES[width]
    mlp = {"kind": "dense", "ff": s["ff"]}
    gla = {"type": "gla", "mixer": {"heads": s["gla"], "dim": 128, "vdim": width // s["gla"], "tau": 16.0}, "mlp": mlp}
    delta = {"type": "channel_delta", "mixer": {"heads": s["delta"], "kv_heads": s["delta"], "dim": 128, "vdim": 128, "conv": 4}, "mlp": mlp}
    att = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": 128, "vdim": 128, "mask": {"size": 512}, "scale": 128 ** -0.5, "softcap": 30.0,
           "rot": {"dims": 128, "base": 10000.0, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    att0, att1 = {"type": "attention", "mixer": att, "mlp": mlp}, {"type": "attention", "mixer": {**att, "kv_from": 2}, "mlp": mlp}
    return {"architecture": "Rurunex", "embedding": {"scale": width ** 0.5}, "layers": [gla, delta, att0, gla, delta, att1, gla, delta, att1], "norm": {"eps": 1e-6}, "logit_scale": 0.5,
            "vocab": vocab, "width": width}


def _timed(fn, iters, warmup=3):
    lib = _lib.load()
    for _ in range(warmup):
        fn()
    gpu.synchronize()
    lib.applegpu_timer_start()
    for _ in range(iters):
        fn()
    return float(lib.applegpu_timer_stop_ms()) / iters


def _kernel_rows(peaks, calls):
    out = {}
    for name, r in sorted(gpu.profile_report().items(), key=lambda kv: -kv[1]["ms"]):
        us, mem = r["ms"] / r["launches"] * 1e3, name in BYTES
        rate = r["work"] / (r["ms"] * 1e-3) if r["ms"] else 0.0
        peak = peaks["hbm_gbs"] * 1e9 if mem else peaks["bf16_tflops"] * 1e12
        out[name] = {"per_step": r["launches"] / calls, "us": round(us, 2), "rate": f"{rate / 1e9:.0f} GB/s" if mem else f"{rate / 1e12:.0f} TFLOP/s", "frac": round(rate / peak, 3)}
    return out


def bench_gedenex(width, peaks, iters=10):
    cfg = config_of(width)
    return bench_sequence(load_gedenex(cfg, init_gedenex_weights(cfg, seed=0), "bfloat16"), width, peaks, iters)


def bench_rurunex(width, peaks, iters=10):
    cfg = rurunex_config_of(width)
    return bench_sequence(load_rurunex(cfg, init_rurunex_weights(cfg, seed=0, ranks={"channel_delta": 128}), "bfloat16"), width, peaks, iters)


def bench_sequence(model, width, peaks, iters=10, batch=8, prompt=1024, steps=48):
    eng = model.engine(slots=batch, max_len=prompt + 2 * steps + 16)
    rng = np.random.default_rng(1)
    ids = rng.integers(0, model.vocab, (batch, prompt)).astype(np.int32)

    def prefill(n=batch):
        eng.reset(0, n)
        eng.forward(ids[:n], logits=False, pick=True)

    row = {"width": width, "layer_runs": 9, "batch": batch, "prompt": prompt}
    ms = _timed(prefill, iters)
    row["prefill_ms"], row["prefill_tokens_per_s"] = round(ms, 3), round(batch * prompt / ms * 1e3)
    gpu.profile(True)
    prefill()
    gpu.profile(False)
    row["prefill_kernels"] = _kernel_rows(peaks, 1)
    for n in (1, batch):
        prefill(n)
        eng.decode(4, 0, n)
        ms = _timed(lambda: eng.decode(steps, 0, n), 1, 0) / steps
        row[f"decode_b{n}_ms"], row[f"decode_b{n}_tokens_per_s"] = round(ms, 4), round(n / ms * 1e3)
        row["decode_launches"], row["decode_graph"] = eng.launches_per_step, eng.uses_graph
        prefill(n)
        gpu.profile(True)
        eng.decode(4, 0, n, use_graph=False)
        gpu.profile(False)
        row[f"decode_b{n}_kernels"] = _kernel_rows(peaks, 4)
        bytes_ = sum(r["work"] for r in gpu.profile_report().values()) / 4      # weights, states and caches a step has to read
        row[f"decode_b{n}_frac"] = round(bytes_ / (row[f"decode_b{n}_ms"] * 1e-3) / peaks["hbm_gbs"] / 1e9, 3)
    eng.close()
    return row


def bench_gpt2(width, peaks, iters=10, batch=8, prompt=1024, steps=48, vocab=32768, layers=9):
    cfg = {"n_layer": layers, "n_head": width // 64, "n_embd": width, "vocab_size": vocab, "n_positions": prompt + 2 * steps + 16}
    model = init_gpt2_weights(cfg, seed=0, dtype="bfloat16")
    ids = np.random.default_rng(1).integers(0, vocab, (batch, prompt))
    keep = {}

    def prefill(n=batch):
        logits, kv = gpt2_forward(model, ids[:n], last_only=True, compiled=True)
        tok = gpu.argmax(logits)
        del logits
        tok.to_numpy()
        keep["kv"], keep["tok"] = kv, tok

    row = {"width": width, "layers": layers, "batch": batch, "prompt": prompt}
    ms = _timed(prefill, iters)
    row["prefill_ms"], row["prefill_tokens_per_s"] = round(ms, 3), round(batch * prompt / ms * 1e3)
    gpu.profile(True)
    prefill()
    gpu.profile(False)
    kern = {}
    for name, r in gpu.profile_report().items():
        if name.startswith(("fused_attention", "fused_linear", "matmul")):
            work = r["launches"] * 2.0 * batch * width * prompt * (prompt + 1) if name.startswith("fused_attention") else r["work"]      # the unmasked half
            rate = work / (r["ms"] * 1e-3)
            kern[name] = {"launches": r["launches"], "us": round(r["ms"] / r["launches"] * 1e3, 2), "rate": f"{rate / 1e12:.0f} TFLOP/s", "frac": round(rate / peaks["bf16_tflops"] / 1e12, 3)}
    row["prefill_kernels"] = kern
    for n in (1, batch):
        prefill(n)
        dec = Gpt2Decoder(model, n, cfg["n_positions"])
        dec.prefill(keep["kv"], keep["tok"], prompt)
        dec.steps(4)
        ms = _timed(lambda: dec.steps(steps), 1, 0) / steps
        bytes_ = 2.0 * (layers * 12 * width * width + vocab * width) + 2.0 * 2 * layers * n * prompt * width
        row[f"decode_b{n}_ms"], row[f"decode_b{n}_tokens_per_s"] = round(ms, 4), round(n / ms * 1e3)
        row[f"decode_b{n}_frac"] = round(bytes_ / (ms * 1e-3) / peaks["hbm_gbs"] / 1e9, 3)
        dec.close()
    return row


def run(peaks, widths=(1024, 2048), iters=10, design="gedenex"):
    """The design at each width beside the closest existing model of equal size: GPT-2 for Gedenex, Gedenex for Rurunex."""
    gpu.init_backend()
    out = []
    t0 = time.time()
    for w in widths:
        if design == "gedenex":
            out.append({"gedenex": bench_gedenex(w, peaks, iters), "gpt2_equal_size": bench_gpt2(w, peaks, iters)})
        else:
            out.append({"rurunex": bench_rurunex(w, peaks, iters), "gedenex_equal_size": bench_gedenex(w, peaks, iters)})
    st = gpu.pipeline_status()
    if st:
        raise RuntimeError(f"pipeline status {st}")
    return {"sizes": out, "seconds": round(time.time() - t0, 1)}
