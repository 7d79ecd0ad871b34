"""Model registry: configuration and engine of every model family, by the ``architecture`` of a ``config.json`` or by the
name of a preset."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, fields
from typing import Any, Callable, Mapping, Optional

import torch

from ..config import HybridConfig, LlamaConfig


@dataclass(frozen=True)
class Family:
    prefix: str                                     # preset names start with it
    named: Callable[..., Any]                       # preset name -> config
    from_dict: Callable[[Mapping[str, Any]], Any]   # config.json -> config
    dtypes: tuple                                   # what the engine computes in
    sources: tuple                                  # kernel sources the inference engine on one GPU needs


def _llama_from_dict(c: Mapping[str, Any]) -> LlamaConfig:
    known = {f.name for f in fields(LlamaConfig)}
    return LlamaConfig(**{k: v for k, v in c.items() if k in known})


FAMILIES = {
    "Llama": Family("llama", LlamaConfig.named, _llama_from_dict, (torch.bfloat16,),
                    ("attn_fwd_sm100", "decode_sm100", "elementwise", "gemm_sm100")),
    "Dafelorn": Family("dafelorn", HybridConfig.named, HybridConfig.from_dict, (torch.bfloat16, torch.float32),
                       ("attn_fwd_sm100", "decode_sm100", "delta_chunk_sm100", "delta_sm100", "gemm_sm100",
                        "latent_decode_sm100", "latent_sm100", "linear_f32", "residual_f32")),
    "Kalonex": Family("kalonex", HybridConfig.named, HybridConfig.from_dict, (torch.bfloat16, torch.float32),
                      ("attn_fwd_sm100", "decode_sm100", "gemm_sm100", "linear_f32", "moe", "moe_gemm_sm100",
                       "residual_f32", "window_decode_sm100", "window_sm100")),
}


def family_of(cfg) -> Family:
    return FAMILIES[cfg.architecture if isinstance(cfg, HybridConfig) else "Llama"]


def load_config(spec: str, **over):
    """``spec``: a preset name, or a folder with a ``config.json``."""
    if os.path.isdir(spec):
        with open(os.path.join(spec, "config.json")) as f:
            c = json.load(f)
        arch = c.get("architecture")
        if arch not in FAMILIES:
            raise ValueError(f"{spec}: unknown architecture {arch!r}; have {sorted(FAMILIES)}")
        if over:
            raise ValueError("a model folder takes no overrides")
        return FAMILIES[arch].from_dict(c)
    for fam in FAMILIES.values():
        if spec.startswith(fam.prefix):
            return fam.named(spec, **over)
    raise KeyError(f"unknown model {spec!r}")


def checkpoint_source(spec: str):
    """Tensor source of a model folder, or None for a preset (random weights)."""
    if not os.path.isdir(spec):
        return None
    from .weights import SafetensorsFile

    return SafetensorsFile(os.path.join(spec, "model.safetensors"))


def make_engine(cfg, max_context: int, *, source=None, dtype: torch.dtype = torch.bfloat16, batch: int = 1, device="cuda",
                seed: int = 0, axis=None, streams: int = 0, max_new_tokens: int = 512, max_step: int = 8192):
    """The inference engine of a configuration. ``source``: tensor name -> tensor (random weights when None). A context
    is rounded up to what the engine needs. ``max_step``: tokens of a sequence that a hybrid decoder with windowed attention
    runs at once."""
    if dtype not in family_of(cfg).dtypes:
        raise ValueError(f"this model does not run in {dtype}")
    if isinstance(cfg, HybridConfig):
        if axis is not None and axis.size > 1:
            raise ValueError("hybrid decoders run on one GPU per engine")
        if streams:
            raise ValueError("hybrid decoders have no shared-prefix streams")
        from .hybrid_infer import HybridInference

        return HybridInference(cfg, max_context, batch=batch, device=device, seed=seed, dtype=dtype, max_step=max_step,
                               source=None if source is None else source.__getitem__)
    from .llama_infer import LlamaInference
    from .params import FlatParams

    unit = 128 * (1 if axis is None else axis.size)
    params: Optional[FlatParams] = None
    if source is not None:
        params = FlatParams(cfg, device, seed, with_optimizer=False)
        for name in params.index:
            params.w(name).copy_(source[name])
    return LlamaInference(cfg, (max_context + unit - 1) // unit * unit, batch=batch, device=device, seed=seed, axis=axis,
                          params=params, streams=streams, max_new_tokens=max_new_tokens)
