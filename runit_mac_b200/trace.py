"""Replays a trace of token portions through a model, step by step, and writes the logits that the trace asks for.

Steps arrive as JSON lines: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  The tokens of an entry extend
the sequence of that id; `want` are places among them whose logits are written to OUT/<step>.f32 (f32, [wanted][vocab], in the
order of the entries and of `want`).  `end` names the sequences that are finished after the step.  A line "done <step>" follows
every step.  The decoder holds one sequence at a time, like everything else that drives it here."""
from __future__ import annotations

import json
import sys
from pathlib import Path

import numpy as np


def replay(model, lines, out_dir, report) -> None:
    out_dir = Path(out_dir)
    live, length = None, 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            if live is None:
                live, length = e["id"], 0
            if e["id"] != live:
                raise ValueError("sequence %r starts before %r has ended" % (e["id"], live))
            if e["tokens"]:
                rows.append(model.forward(e["tokens"], length, e["want"]))
                length += len(e["tokens"])
        if sum(len(r) for r in rows):
            np.concatenate(rows).astype("<f4").tofile(out_dir / ("%d.f32" % step["step"]))
        if live in step.get("end", ()):
            live = None
        report("done %d" % step["step"])


def run(model_dir, dtype: str, out_dir, max_tokens: int) -> int:
    from . import _lib, build
    _lib.load(build.ensure("layered"))
    from . import dispatch, models
    ctx = dispatch.Context(0)
    model = models.load_model(ctx, model_dir, dtype, max_seq=max(int(max_tokens), 16))
    replay(model, iter(sys.stdin.readline, ""), out_dir, lambda s: print(s, flush=True))
    model.close()
    ctx.close()
    return 0
