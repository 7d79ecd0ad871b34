#!/usr/bin/env python
"""Long-context inference entry point: chunked prefill into a sequence-sharded KV cache, then
greedy decoding. Reports prefill tokens/s, decode tokens/s and p50 per-token latency as JSON.

    python infer.py --model llama-7b --context 131072 --new-tokens 64
    python -m torch.distributed.run --nproc-per-node 8 --master-addr 127.0.0.1 infer.py \
        --model llama-7b --context 1048576 --chunk 32768 --new-tokens 256 --batch 1
    ... --streams 4      # four decode streams that share the one cached context
    python infer.py --model dafelorn-7b --context 131072 --new-tokens 64
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import sys

os.environ.setdefault("PYTORCH_CUDA_ALLOC_CONF", "expandable_segments:True")
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))


def main() -> int:
    ap = argparse.ArgumentParser(description=__doc__.splitlines()[0])
    ap.add_argument("--model", default="llama-7b",
                    help="a preset (llama-*, dafelorn-*, kalonex-*) or a folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="float32: hybrid decoders only")
    ap.add_argument("--context", type=int, default=131072, help="tokens of cached context to prefill")
    ap.add_argument("--chunk", type=int, default=32768)
    ap.add_argument("--new-tokens", type=int, default=256)
    ap.add_argument("--batch", type=int, default=1)
    ap.add_argument("--streams", type=int, default=0,
                    help="decode this many streams (<= 8) from ONE cached context (batch must be 1): the way a batch of "
                         "long-context requests fits when distinct contexts do not")
    ap.add_argument("--layers", type=int, default=None, help="override layer count (debug)")
    args = ap.parse_args()

    import torch
    import torch.distributed as dist

    from ringattention_b200.config import HybridConfig
    from ringattention_b200.models import registry
    from ringattention_b200.ops import _lib
    from ringattention_b200.parallel.mesh import DeviceMesh
    from ringattention_b200.trainer import init_distributed

    rank, world, local = init_distributed()
    mesh = DeviceMesh(f"1,1,1,{world}")
    over = {} if args.layers is None else {"n_layers": args.layers}
    cfg = registry.load_config(args.model, **over)
    dev = torch.device("cuda", local)
    max_ctx = (args.context + args.new_tokens + 128 * world - 1) // (128 * world) * (128 * world)
    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[args.dtype]
    if isinstance(cfg, HybridConfig):
        kv_gb = args.batch * cfg.cache_bytes(max_ctx, dtype.itemsize, max_step=8192) / 1e9
    else:
        kv_gb = args.batch * max_ctx / world * 2 * cfg.d_model * 2 * cfg.n_layers / 1e9
    free_gb = torch.cuda.mem_get_info(dev)[0] / 1e9
    if kv_gb + cfg.n_params() * dtype.itemsize / 1e9 > free_gb * 0.95:
        if rank == 0:
            print(json.dumps({"error": "KV cache does not fit", "kv_cache_gb_per_gpu": kv_gb,
                              "free_gb": free_gb, "batch": args.batch, "context": args.context}))
        return 0
    source = registry.checkpoint_source(args.model)
    eng = registry.make_engine(cfg, max_ctx, source=source, dtype=dtype, batch=args.batch, device=dev,
                               axis=mesh.axis("sp"), streams=args.streams, max_new_tokens=args.new_tokens + 8)
    g = torch.Generator().manual_seed(0)
    prompt = torch.randint(0, cfg.vocab_size, (args.batch, args.context), generator=g)
    gen, timing = eng.generate(prompt.to(dev), args.new_tokens, chunk=args.chunk)
    _lib.check_status(dev)
    lat = timing["decode_ms"]
    # the first steps run eagerly and record the CUDA graph; throughput is quoted on the replayed steps
    steady = lat[3:] if len(lat) > 6 else lat
    t = torch.tensor([timing["prefill_s"], sum(steady) / 1e3], device=dev, dtype=torch.float64)
    if world > 1:
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
    if rank == 0:
        print(json.dumps({
            "model": args.model, "n_layers": cfg.n_layers, "n_gpus": world, "batch": args.batch,
            "context": args.context, "chunk": args.chunk, "new_tokens": args.new_tokens,
            "prefill_tokens_per_s": args.batch * args.context / float(t[0]),
            "decode_tokens_per_s": max(args.batch, args.streams) * len(steady) / float(t[1]),
            "streams_sharing_the_context": args.streams,
            "decode_first_steps_ms": [round(x, 3) for x in lat[:3]],
            "decode_p50_ms": statistics.median(steady), "decode_p90_ms": sorted(steady)[int(0.9 * (len(steady) - 1))],
            "kv_cache_gb_per_gpu": kv_gb,
            "data": "random tokens, " + ("random-init weights" if source is None else "weights of the model folder"),
            "dtype": "bf16" if args.dtype == "bfloat16" else "fp32"}))
    if world > 1:
        dist.barrier()
        dist.destroy_process_group()
    return 0


if __name__ == "__main__":
    sys.exit(main())
