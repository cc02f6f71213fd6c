"""Trace replay: feeds given token ids through a model step by step and writes the logits that are asked for.

Each line of standard input is one step, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: the next tokens of
each request, the places among them whose logits are wanted, and the requests that are finished afterwards. A step with
wanted places leaves OUT/<step>.f32 (little-endian float32 [wanted, vocab], in the order of the entries); every step is
answered with a line "done <step>". Nothing is sampled; the steps run on the engine that generation uses.
"""
import argparse
import json
import os
import sys

import numpy as np

SLOTS = 2


class Replay:
    def __init__(self, model, max_tokens):
        self.model = model
        self.engine = model.engine(slots=SLOTS, max_len=max(int(max_tokens), 1))
        self.slot_of = {}

    def step(self, entries, end):
        """Logits [wanted, vocab] of one step, None if nothing is wanted."""
        got = []
        for e in entries:
            if e["id"] not in self.slot_of:
                self.slot_of[e["id"]] = self.engine.acquire()
            if not e["tokens"]:
                continue
            want = e.get("want") or []
            logits, _ = self.engine.forward(e["tokens"], slot=self.slot_of[e["id"]], want=want, logits=bool(want))
            if want:
                got.append(logits)
        for r in end:
            if r in self.slot_of:
                self.engine.release(self.slot_of.pop(r))
        return np.concatenate(got) if got else None


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096)
    a = ap.parse_args(argv)

    from . import api as gpu
    from .models import load_model
    from .seqmodel import SequenceModel
    gpu.init_backend()
    model = load_model(a.model, a.dtype)
    if not isinstance(model, SequenceModel):
        print("trace replay runs sequence models only", file=sys.stderr)
        return 2
    replay = Replay(model, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s.get("entries", []), s.get("end", []))
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
