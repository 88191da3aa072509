"""Trace replay: given token ids go through a model step by step and the logits that are asked for are written out.

Steps come as JSON lines on standard input, ``{"step": s, "entries": [{"id", "tokens", "want"}], "end": [ids]}``.  All entries of
a step are one rows step of the engine; ids are bound to lanes at their first entry and leave them when they end.  For a step
with wanted places ``<out>/<step>.f32`` holds their logits (little-endian float32, [wanted, vocab], in the order of the entries);
``done <step>`` is printed after every step.
"""
from __future__ import annotations

import json
import os
import sys

LANES = 4


def run(args, inp=None, out=None) -> int:
    inp, out = inp or sys.stdin, out or sys.stdout
    from ..kv.paged import PAGE
    from ..models import registry
    pool = -(-args.max_tokens // PAGE) * PAGE
    eng = registry.layered_engine(args.model, args.dtype, max_context=pool, max_lanes=LANES, max_rows=min(pool, 65535), pool_tokens=pool)
    lane_of: dict[str, int] = {}
    at: dict[str, int] = {}
    for line in inp:
        if not line.strip():
            continue
        msg = json.loads(line)
        tokens, lanes, positions, want = [], [], [], []
        for e in msg["entries"]:
            rid = e["id"]
            if rid not in lane_of:
                free = [k for k in range(LANES) if k not in lane_of.values()]
                if not free:
                    raise RuntimeError(f"more than {LANES} live requests")
                lane_of[rid], at[rid] = free[0], 0
            want += [len(tokens) + k for k in e["want"]]
            tokens += e["tokens"]
            lanes += [lane_of[rid]] * len(e["tokens"])
            positions += range(at[rid], at[rid] + len(e["tokens"]))
            at[rid] += len(e["tokens"])
        if tokens:
            # a step of single tokens takes the head on every row (the captured decode step); otherwise only the wanted rows
            single = len(set(lanes)) == len(lanes)
            eng.step(tokens, lanes, positions, head=True if single else want, sample=False)
            if want:
                logits = eng.logits[want] if single else eng.logits
                data = logits.float().cpu().numpy().astype("<f4").tobytes()
                path = os.path.join(args.out, f"{msg['step']}.f32")
                with open(path + ".part", "wb") as f:
                    f.write(data)
                os.replace(path + ".part", path)
            eng.check_status()
        for rid in msg.get("end", []):
            if rid in lane_of:
                eng.release_lane(lane_of.pop(rid))
                at.pop(rid)
        print(f"done {msg['step']}", file=out, flush=True)
    return 0
