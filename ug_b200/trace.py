"""Trace replay: feeds given token ids through a model step by step and writes the logits that are asked for.

Steps are JSON lines on standard input:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}
A step appends its tokens to the sequence ``id``; the logits at the places ``want`` of those tokens go to
OUT/<step>.f32 (little-endian f32, [wanted, vocab]).  "done <step>" follows on standard output.  ``end`` finishes
sequences; a new one may start after that.  One sequence is live at a time: it is row 0 of a batch of one.
"""
import argparse
import json
import os
import sys

import numpy as np


class Replay:
    def __init__(self, model, out_dir):
        self.model, self.out_dir, self.live = model, out_dir, None

    def feed(self, tokens, want):
        """Appends the tokens; f32 [len(want), vocab]."""
        m, n = self.model, len(tokens)
        if n == 1:
            m.fwd(np.array(tokens, np.int32))
            rows = m.logits() if want else None
        else:
            every = any(k != n - 1 for k in want)
            m.prefill(np.array([tokens], np.int32), all_logits=every)
            if every:
                return m.prefill_logits()[0][list(want)]
            rows = m.logits() if want else None
        return rows[[0] * len(want)] if want else np.empty((0, m.vocab_local), np.float32)

    def step(self, s):
        entries, rows = s.get("entries", []), []
        for e in entries:
            if self.live is None:
                self.model.reset()
                self.live = e["id"]
            elif self.live != e["id"]:
                raise ValueError(f"sequence {e['id']!r} starts while {self.live!r} is live")
            if e["tokens"]:
                rows.append(self.feed(e["tokens"], e.get("want", [])))
        self.model.dev.synchronize()
        if any(e.get("want") for e in entries):
            path = os.path.join(self.out_dir, f"{s['step']}.f32")
            np.concatenate(rows).astype("<f4").tofile(path)
        if self.live in s.get("end", []):
            self.live = None


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replays a token trace and writes logits")
    ap.add_argument("--model", required=True, help="folder with config.json and .safetensors files")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens a live sequence holds")
    a = ap.parse_args(argv)
    from . import registry
    from .device import Device
    from .generate import DTYPES
    dtype = DTYPES[a.dtype]
    if dtype not in registry.DTYPES[registry.architecture(registry.read_config(a.model))]:
        print(f"this model does not run in {a.dtype}", file=sys.stderr)
        return 3
    model = registry.load(a.model, Device(0), 1, max(1, a.max_tokens), dtype)
    replay = Replay(model, a.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        replay.step(s)
        print(f"done {s['step']}", flush=True)
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
