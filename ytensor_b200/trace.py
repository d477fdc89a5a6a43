"""Replays a trace: token ids of requests, fed to a model step by step, logits of chosen places written to files.

Steps are JSON lines on standard input:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
For a step that wants something <out>/<step>.f32 holds the logits in the order asked for (little-endian fp32,
[wanted, vocab]); after every step `done <step>` is printed. A request's tokens are appended to what earlier steps left in
the model's cache; "end" gives the cache back. The model holds one sequence, so requests come one after the other.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path


class Replay:
    """The requests of a trace on one model of one sequence."""

    def __init__(self, model):
        self.model, self.live = model, None

    def step(self, entries, end=()):
        """Runs one step; returns the wanted logits [wanted, vocab] as a numpy array, or None."""
        import numpy as np
        m, torch = self.model, self.model.torch
        out = []
        for e in entries:
            if self.live is None:
                m.reset_kv_cache()
                self.live = e["id"]
            elif self.live != e["id"]:
                raise ValueError("a request begins while another one is running: this model holds one sequence")
            tokens, want = list(e["tokens"]), list(e.get("want", ()))
            if not tokens:
                continue
            ids = torch.tensor([tokens], dtype=torch.int32, device="cuda")
            places = sorted(set(want))
            logits = m.forward_at(ids, places)
            if want:
                at = {p: i for i, p in enumerate(places)}
                out.append(logits.cpu().numpy()[[at[p] for p in want]])
        if self.live in end:
            self.live = None
        m.check_status()
        return np.concatenate(out) if out else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    from .registry import UnsupportedModel, find_model, load_model, read_config
    try:
        entry = find_model(read_config(a.model))
    except UnsupportedModel as e:
        print(e, file=sys.stderr)
        return 2
    if a.dtype not in entry.dtypes:
        print(f"{entry.name} does not run in {a.dtype}", file=sys.stderr)
        return 3
    model = load_model(a.model, dtype=a.dtype, max_tokens=max(1, a.max_tokens), build=True)
    replay = Replay(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s.get("entries", ()), s.get("end", ()))
        if logits is not None:
            path = Path(a.out) / f"{s['step']}.f32"
            part = path.with_suffix(".part")
            part.write_bytes(logits.astype("<f4").tobytes())
            os.replace(part, path)
        print(f"done {s['step']}", flush=True)
    model.close()
    return 0
