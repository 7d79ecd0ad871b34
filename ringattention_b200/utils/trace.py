"""Trace replay: feed given token ids through a model, step by step, and write logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

``DIR`` holds ``config.json`` and ``model.safetensors``. Every line of standard input is one step::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry brings a request's next tokens and the places among them whose logits are wanted; ``end`` names the requests
that are finished after the step. A step in which something is wanted writes ``OUT/<step>.f32`` (the wanted rows in order,
little-endian fp32); after every step a line ``done <step>`` is printed. Requests come one after the other: the engine
holds one sequence, and its cache and states are given back when the request ends. The engine and its step functions are
the ones that generation uses; one token at a time goes through the decode step.

Exit code 3: the model has no engine in the requested type.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Optional

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class TraceRunner:
    def __init__(self, engine):
        self.engine = engine
        self.current: Optional[str] = None

    def entry(self, rid: str, tokens: list, want: list) -> Optional[torch.Tensor]:
        """Run one entry; returns the wanted logits ``(len(want), vocab)``."""
        eng = self.engine
        if self.current != rid:
            if self.current is not None:
                raise ValueError(f"request {rid!r} starts before {self.current!r} has ended")
            eng.reset()
            self.current = rid
        if not tokens:
            raise ValueError("an entry without tokens")
        if any(not 0 <= w < len(tokens) for w in want):
            raise ValueError("want names a place outside the entry")
        tok = torch.tensor([tokens], dtype=torch.int32, device=eng.device)
        if len(tokens) == 1 and eng.length > 0:
            logits = eng.decode_step(tok[0])
            return logits[[0] * len(want)] if want else None
        if hasattr(eng, "step"):
            out = eng.step(tok, want=want)
            return None if out is None else out[0]
        if want and list(want) != [len(tokens) - 1]:
            raise ValueError("this model's engine gives the logits of a step's last token only")
        logits = eng.prefill_chunk(tok)
        return logits if want else None

    def end(self, rid: str) -> None:
        if rid != self.current:
            raise ValueError(f"request {rid!r} is not live")
        self.engine.reset()
        self.current = None

    def step(self, line: dict, out_dir: str) -> None:
        rows = [r for e in line["entries"] for r in [self.entry(e["id"], e["tokens"], e["want"])] if r is not None]
        if rows:
            data = torch.cat(rows).float().cpu().contiguous().numpy().astype("<f4").tobytes()
            with open(os.path.join(out_dir, f"{line['step']}.f32"), "wb") as f:
                f.write(data)
        for rid in line["end"]:
            self.end(rid)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="the most tokens live requests hold at any time")
    args = ap.parse_args(argv)

    from ..models import registry
    from ..ops import _lib

    cfg = registry.load_config(args.model)
    dtype = DTYPES[args.dtype]
    if dtype not in registry.family_of(cfg).dtypes:
        print(f"trace_run: this model does not run in {args.dtype}", file=sys.stderr)
        return 3
    _lib.need_only(registry.family_of(cfg).sources)
    engine = registry.make_engine(cfg, max(1, args.max_tokens), source=registry.checkpoint_source(args.model), dtype=dtype)
    runner = TraceRunner(engine)
    for text in sys.stdin:
        if not text.strip():
            continue
        line = json.loads(text)
        runner.step(line, args.out)
        _lib.check_status(engine.device)
        print(f"done {line['step']}", flush=True)
    return 0
