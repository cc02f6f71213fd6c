"""Command line: `python -m applegpu_runtime_b200 generate --model DIR --prompt 1,2,3 [--prompt ...] --max-tokens 20`.

Prompts and results are token ids. Several prompts (of any lengths, for sequence models) are continued side by side when
greedy; with a temperature they are sampled one after the other.
"""
import argparse
import json
import sys

import numpy as np


def main(argv=None):
    ap = argparse.ArgumentParser(prog="applegpu_runtime_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="continue prompts with a model folder (config.json, model.safetensors)")
    g.add_argument("--model", required=True)
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float16", "float32"])
    g.add_argument("--prompt", action="append", required=True, help="token ids with commas between them; may be given several times")
    g.add_argument("--max-tokens", type=int, default=20)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=50)
    g.add_argument("--top-p", type=float, default=0.9)
    g.add_argument("--seed", type=int, default=None)
    a = ap.parse_args(argv)

    from . import api as gpu
    from .generate import generate, greedy_generate
    from .models import load_model
    gpu.init_backend()
    prompts = [[int(x) for x in p.split(",") if x.strip()] for p in a.prompt]
    model = load_model(a.model, a.dtype)
    if a.temperature <= 0:
        same = len({len(p) for p in prompts}) == 1
        out = greedy_generate(model, prompts, a.max_tokens) if same or not isinstance(model, dict) else [greedy_generate(model, p, a.max_tokens)[0] for p in prompts]
    else:
        if a.seed is not None:
            np.random.seed(a.seed)
        out = [generate(model, p, a.max_tokens, temperature=a.temperature, top_k=a.top_k, top_p=a.top_p) for p in prompts]
    for r in out:
        print(json.dumps([int(x) for x in r]))
    return 0


if __name__ == "__main__":
    sys.exit(main())
