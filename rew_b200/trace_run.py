"""Replays a trace of token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are JSON objects on standard input, one a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

entries: the requests' next tokens and the places among them whose logits are wanted; end: requests that give back
what they hold after the step.  A step is one rewb200_lanes_feed call: all its entries are one batch.  Wanted logits go
to DIR/<step>.f32 (little-endian f32 [wanted, vocab]); "done <step>" follows on standard output.  At most
REQUESTS requests are live at a time, and the pool has the pages --max-tokens asks for.
"""
import argparse
import json
import os
import sys

REQUESTS = 4
PAGE = 64


class Replay:
    """Requests of a trace on the lanes of one paged session."""

    def __init__(self, model, max_tokens):
        import numpy as np
        self.np = np
        pages = max(1, (max_tokens + PAGE - 1) // PAGE)
        self.session = model.paged_session(REQUESTS, pages * PAGE, pages + 1)   # and the idle lanes' scratch page
        self.lanes, self.idle = {}, list(range(REQUESTS))

    def step(self, entries, end):
        """Logits [wanted, vocab] in the order of the entries and of their want."""
        portions, want, order, row0 = [], [], [], 0
        for e in entries:
            if e["id"] not in self.lanes:
                if not self.idle:
                    raise ValueError("more than %d live requests" % REQUESTS)
                self.lanes[e["id"]] = self.idle.pop(0)
            portions.append((self.lanes[e["id"]], e["tokens"]))
            for w in e.get("want", []):
                if not 0 <= w < len(e["tokens"]):
                    raise ValueError("wanted place %d is not among the entry's tokens" % w)
                want.append(row0 + w)
            row0 += len(e["tokens"])
        logits = self.np.empty((0, self.session.model.cfg.vocab), self.np.float32)
        if portions:
            places = sorted(set(want))
            got, _ = self.session.feed(portions, want=places)
            at = {p: i for i, p in enumerate(places)}
            logits = got[[at[w] for w in want]]
        for rid in end:
            lane = self.lanes.pop(rid)
            self.session.release(lane)
            self.idle.append(lane)
        return logits


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds, in pages of %d" % PAGE)
    args = ap.parse_args(argv)
    from . import build
    build.build()                       # compiles what is missing or out of date
    from .models import load_model
    pages = max(1, (args.max_tokens + PAGE - 1) // PAGE)
    replay = Replay(load_model(args.model, dtype=args.dtype, max_seq=pages * PAGE), args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end", []))
        if len(logits):
            with open(os.path.join(args.out, "%d.f32" % step["step"]), "wb") as f:
                f.write(logits.astype("<f4").tobytes())
        print("done %d" % step["step"], flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
