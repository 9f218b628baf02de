"""Replays a trace of given tokens through an engine, step by step, and writes the logits that the trace asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

DIR holds config.json and model.safetensors.  Steps are JSON objects, one per line of standard input::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry brings a request's next tokens and the places among them whose logits are wanted; all entries of a step run as
one batch (`Engine.step`), whatever their lengths.  Requests are admitted at their first entry and release their pages
and state slot when "end" names them.  A step with wanted places writes DIR/<step>.f32 ([wanted, vocab], little-endian
fp32, in the order of the entries); after every step the line "done <step>" is printed.

The KV pool holds N tokens in pages of 64, and there are state slots for four requests.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Optional

import numpy as np
import torch

DTYPES = {"bfloat16": torch.bfloat16, "float16": torch.float16, "float32": torch.float32}
PAGE = 64
LIVE_REQUESTS = 4


class TraceRunner:
    def __init__(self, model: str, dtype: torch.dtype, max_tokens: int, max_batch: int = 64, max_batch_tokens: int = 4096):
        from . import core
        from .engine import Engine
        self.core = core
        self.engine = Engine(model, num_pages=max(1, -(-max_tokens // PAGE)), page_size=PAGE, max_batch=max_batch,
                             max_batch_tokens=max_batch_tokens, dtype=dtype, ready=False, state_slots=LIVE_REQUESTS)
        self.engine.load_checkpoint(model)
        self.batch = core.Batch(0, self.engine.pool, self.engine.slots)
        self.ids: Dict[str, int] = {}
        self.next_id = 0

    def _bring(self, name: str, tokens) -> int:
        """Admit or extend a request; its number."""
        if name in self.ids:
            ok = self.batch.extend_prompt(self.ids[name], tokens)
        else:
            self.ids[name] = self.next_id
            self.next_id += 1
            ok = self.batch.add_prompts([self.core.SeqSpec(self.ids[name], tokens, 1)], False)
        if not ok:
            raise RuntimeError(f"request {name!r}: no free pages or state slots")
        return self.ids[name]

    def step(self, entries, end) -> Optional[np.ndarray]:
        """Logits [wanted, vocab] in the order of the entries, or None."""
        from .. import ops
        got = None
        entries = [e for e in entries if e["tokens"]]
        if entries:
            seen = [self._bring(e["id"], list(e["tokens"])) for e in entries]
            order = self.batch.request_ids()
            counts, want, place = [0] * len(order), [[] for _ in order], []
            for e, i in zip(entries, seen):
                at = order.index(i)
                counts[at] = len(e["tokens"])
                want[at] = list(e.get("want", []))
            logits = self.engine.step(self.batch, counts, want)
            if logits is not None:
                starts = np.concatenate([[0], np.cumsum([len(w) for w in want])])
                for i in seen:
                    at = order.index(i)
                    place += range(int(starts[at]), int(starts[at + 1]))
                got = logits.cpu().numpy()[place]
            ops.check_status()
        gone = {self.ids.pop(n) for n in end if n in self.ids}
        if gone:
            self.batch.filter([i for i in self.batch.request_ids() if i not in gone])
        return got


def main(argv=None) -> int:
    ap = argparse.ArgumentParser("trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=list(DTYPES))
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    os.makedirs(a.out, exist_ok=True)
    runner = TraceRunner(a.model, DTYPES[a.dtype], a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = runner.step(s["entries"], s.get("end", []))
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
