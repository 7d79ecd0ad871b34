"""Serving benchmark of hybrid decoders beside the LLaMA engine at equal width, depth and feed-forward parameters.

    python bench.py --serve [--serve-models dafelorn-1b,dafelorn-7b,kalonex-1b,kalonex-7b] [--serve-layers 8] ...
    python -m ringattention_b200.utils.servebench --kernels          # device time per launcher of one prefill chunk

A model whose layers run several times counts layer runs. For every model: prefill tokens/s (chunks of ``--chunk`` tokens up to ``--context``) and decode tokens/s at that context
(replayed CUDA graph), with random weights and tokens. All device times are CUDA events. The working set of a step (the
weights) exceeds the L2 by far, so no flush is needed between steps.
"""
from __future__ import annotations

import argparse
import json
import statistics
from collections import defaultdict

import torch

PARTNER = {f"{d}-{n}": f"llama-{n}" for d in ("dafelorn", "kalonex") for n in ("tiny", "1b", "7b")}


def build(model: str, layers, max_context: int, batch: int):
    from ..models import registry

    cfg = registry.load_config(model, **({} if layers is None else {"n_layers": layers}))
    return cfg, registry.make_engine(cfg, max_context, batch=batch)


def n_runs(cfg) -> int:
    return len(cfg.runs) if hasattr(cfg, "runs") else cfg.n_layers


def run_model(model: str, layers, context: int, chunk: int, batch: int, new_tokens: int, warmup: int = 3) -> dict:
    from ..ops import _lib

    cfg, eng = build(model, layers, context + new_tokens + 128, batch)
    g = torch.Generator().manual_seed(0)
    prompt = torch.randint(0, cfg.vocab_size, (batch, context), generator=g).cuda()
    for _ in range(warmup):
        eng.prefill_chunk(prompt[:, :chunk])
        eng.reset()
    ev = lambda: torch.cuda.Event(enable_timing=True)
    e0, e1 = ev(), ev()
    torch.cuda.synchronize()
    e0.record()
    for c0 in range(0, context, chunk):
        logits = eng.prefill_chunk(prompt[:, c0:c0 + chunk])
    e1.record()
    torch.cuda.synchronize()
    prefill_ms = e0.elapsed_time(e1)
    nxt = eng.sample(logits)
    for _ in range(2):
        nxt = eng.sample(eng.decode_step(nxt))
    eng._tok_buf.copy_(nxt.to(torch.int32))
    for _ in range(warmup):
        eng.decode_step_graph()
    lat = []
    for _ in range(new_tokens - warmup - 2):
        a, b = ev(), ev()
        a.record()
        eng.decode_step_graph()
        b.record()
        torch.cuda.synchronize()
        lat.append(a.elapsed_time(b))
    _lib.check_status()
    ms = statistics.median(lat)
    out = {"model": model, "n_layers": n_runs(cfg), "params_b": round(cfg.n_params() / 1e9, 3), "batch": batch,
           "context": context, "chunk": chunk, "prefill_tokens_per_s": round(batch * context / prefill_ms * 1e3),
           "prefill_ms": round(prefill_ms, 2), "decode_ms": round(ms, 4), "decode_tokens_per_s": round(batch / ms * 1e3, 1),
           "decode_steps": len(lat)}
    del eng
    torch.cuda.empty_cache()
    return out


class CallTimer:
    """Device time per launcher: CUDA events around every call of the kernel library (for GPU-bound steps)."""

    def __enter__(self):
        from ..ops import _lib

        self.lib, self.orig, self.ev = _lib, _lib.call, []

        def call(name, *args, **kw):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            self.orig(name, *args, **kw)
            b.record()
            shape = tuple(x for x in args[5:8]) if name == "ra_gemm_bf16_ex" else (
                tuple(x for x in args[4:7]) if name == "ra_gemm_bf16" else ())
            self.ev.append((name, shape, a, b))

        _lib.call = call
        return self

    def __exit__(self, *exc):
        self.lib.call = self.orig
        torch.cuda.synchronize()
        acc = defaultdict(list)
        for name, shape, a, b in self.ev:
            acc[name + (str(list(shape)) if shape else "")].append(a.elapsed_time(b))
        self.rows = {k: {"calls": len(v), "ms_total": round(sum(v), 3), "ms_median": round(statistics.median(v), 4)}
                     for k, v in acc.items()}


def kernels(model: str, layers, context: int, chunk: int, batch: int) -> dict:
    """Per-launcher device times of the last prefill chunk of a ``context``-token prompt and of one eager decode step."""
    cfg, eng = build(model, layers, context + 128, batch)
    prompt = torch.randint(0, cfg.vocab_size, (batch, context), generator=torch.Generator().manual_seed(0)).cuda()
    for _ in range(3):
        for c0 in range(0, context - chunk, chunk):
            eng.prefill_chunk(prompt[:, c0:c0 + chunk])
        with CallTimer() as t:
            logits = eng.prefill_chunk(prompt[:, context - chunk:])
        nxt = eng.sample(logits)
        eng.decode_step(nxt)
        with CallTimer() as d:
            eng.decode_step(nxt)
        eng.reset()
    return {"model": model, "context": context, "chunk": chunk, "batch": batch, "n_layers": n_runs(cfg),
            "prefill_chunk": t.rows, "decode_step_eager": d.rows}


def add_arguments(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--serve-models", default="dafelorn-1b,dafelorn-7b,kalonex-1b,kalonex-7b",
                    help="hybrid presets; each is followed by the LLaMA preset of equal size")
    ap.add_argument("--serve-layers", type=int, default=None, help="override the number of layer runs (a multiple of 4)")
    ap.add_argument("--serve-context", type=int, default=32768)
    ap.add_argument("--serve-chunk", type=int, default=8192)
    ap.add_argument("--serve-batches", default="1,4")
    ap.add_argument("--serve-new-tokens", type=int, default=64)


def main(args) -> int:
    from .metrics import device_memory_used_gb  # noqa: F401  (fails early without a device)

    rows = []
    for model in args.serve_models.split(","):
        for b in [int(x) for x in args.serve_batches.split(",")]:
            for m in [model] + ([PARTNER[model]] if model in PARTNER else []):
                rows.append(run_model(m, args.serve_layers, args.serve_context, args.serve_chunk, b, args.serve_new_tokens))
    print(json.dumps({"metric": "prefill and decode tokens/s of the inference engines", "n_gpus": 1, "dtype": "bf16",
                      "data": "random tokens, random-init weights", "rows": rows}))
    return 0


if __name__ == "__main__":
    ap = argparse.ArgumentParser(description=__doc__.splitlines()[0])
    add_arguments(ap)
    ap.add_argument("--kernels", action="store_true", help="device time per launcher instead")
    a = ap.parse_args()
    if a.kernels:
        for mdl in a.serve_models.split(","):
            for bb in a.serve_batches.split(","):
                print(json.dumps(kernels(mdl, a.serve_layers, a.serve_context, a.serve_chunk, int(bb))))
    else:
        raise SystemExit(main(a))
