"""Replay a trace: feed given token ids through a model step by step and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A line of standard input describes one step of the engine:

    {"step": 7, "entries": [{"id": "q1", "tokens": [812], "want": [0]}, {"id": "q2", "tokens": [4, 4, 90], "want": []}], "end": ["q1"]}

All entries go through the model in one batch, prompt portions of any length next to single tokens.  ``want`` lists places
in an entry's tokens; their logits are stored in OUT/<step>.f32 as fp32 rows, entry by entry (a step that wants none leaves
no file).  The cache blocks of the requests in ``end`` are freed once the step has run, and ``done <step>`` is printed.

The tool is a thin client of the continuous-batching API: a request's first entry is admitted with `set_input_cb`, later
ones continue it (`extend=True`), `forward_cb` runs the step, `free_seqs` ends requests.  Nothing is sampled.  The KV pools
are made once for ``--max-tokens`` tokens, pools of recurrent states for MAX_SEQUENCES requests.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict

MAX_SEQUENCES = 4                 # live requests a trace may hold
DTYPES = {"bfloat16": "bf16", "float32": "fp32"}


class TraceRunner:
    def __init__(self, path: str, dtype: str, max_tokens: int, max_sequences: int = MAX_SEQUENCES):
        import torch

        from ..automodel import AutoModel
        from ..utils.flags import Env
        if not torch.cuda.is_available() and not Env.get().engine.upper().startswith("CPU"):
            raise RuntimeError("no CUDA device (XFT_ENGINE=CPU runs the PyTorch path)")
        self.model = AutoModel.from_pretrained(path, dtype=dtype, kv_cache_dtype="bf16", max_cache_tokens=max_tokens,
                                               max_sequences=max_sequences)
        self.ids: Dict[str, int] = {}

    def step(self, entries, end=()):
        """Run one step; returns the wanted logits [rows, vocab] on the host (possibly no rows)."""
        m = self.model
        new = [e for e in entries if e["id"] not in self.ids]
        old = [e for e in entries if e["id"] in self.ids]
        if new:
            got = m.set_input_cb([e["tokens"] for e in new], max_length=1 << 30, hold=bool(old),
                                 rows=[e.get("want", []) for e in new], on_demand=True)
            self.ids.update({e["id"]: int(s) for e, s in zip(new, got)})
        if old:
            m.set_input_cb([e["tokens"] for e in old], [self.ids[e["id"]] for e in old], extend=True, append=bool(new),
                           rows=[e.get("want", []) for e in old])
        logits = None
        if entries:
            logits = m.forward_cb().float().cpu()
            if m.model.ctx.device.type == "cuda":
                from ..ops import native
                native.Workspace.get(m.model.ctx.device).check_status()
            # the batch holds the new requests first: back to the order of the entries
            spans, at = {}, 0
            for e in new + old:
                spans[e["id"]] = range(at, at + len(e.get("want", [])))
                at += len(e.get("want", []))
            logits = logits[[r for e in entries for r in spans[e["id"]]]]
        if end:
            m.free_seqs([self.ids.pop(i) for i in end if i in self.ids])
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="model directory")
    ap.add_argument("--dtype", required=True, choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="directory of the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the KV pools in tokens")
    a = ap.parse_args(argv)
    r = TraceRunner(a.model, DTYPES[a.dtype], a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = r.step(s.get("entries", []), s.get("end", []))
        if logits is not None and logits.shape[0]:
            part = os.path.join(a.out, f".{s['step']}.part")
            logits.numpy().astype("<f4").tofile(part)
            os.replace(part, os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
