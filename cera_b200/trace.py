"""Trace replay: token ids in, step by step, logits out (bin/trace_run)."""
import argparse
import json
import os
import sys

import numpy as np

from .registry import load_model


class TraceRunner:
    """Feeds a model's one sequence: a request starts on an empty state and holds it until it ends."""

    def __init__(self, model):
        self.model = model
        self.live = None

    def step(self, entries):
        """-> float32 [wanted places of all entries, vocab]"""
        rows = []
        for e in entries:
            if self.live is None:
                self.model.truncate_kv(0)
                self.live = e["id"]
            elif e["id"] != self.live:
                raise RuntimeError(f"request {e['id']!r} begins before {self.live!r} has ended: the model holds one sequence")
            rows.append(self.model.forward_prefill_logits_at(e["tokens"], self.model.seq_len, e["want"]))
        return np.concatenate(rows) if rows else np.empty((0, self.model.cfg.vocab_size), dtype=np.float32)

    def end(self, ids):
        if self.live in ids:
            self.model.truncate_kv(0)
            self.live = None


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="longest sequence the trace holds")
    a = ap.parse_args(argv)
    model = load_model(a.model, dtype=a.dtype, max_seq_len=max(a.max_tokens, 1))
    run = TraceRunner(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        out = run.step(s["entries"])
        if len(out):
            with open(os.path.join(a.out, f"{s['step']}.f32"), "wb") as f:
                f.write(np.ascontiguousarray(out, dtype="<f4").tobytes())
        run.end(s.get("end", []))
        print(f"done {s['step']}", flush=True)
    model.close()
    return 0
