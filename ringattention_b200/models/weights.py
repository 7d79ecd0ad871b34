"""Weight loading: a reader of ``model.safetensors`` files and the packed weights of hybrid decoders.

Packing puts what a step reads together: the input projections of a mixer are one matrix (segments start at multiples of
eight rows so that every part of the product is 16-byte aligned), the mixer's and the feed-forward's output projections
are one matrix side by side where both read the same stream (their sum is one product over the concatenated inputs), gate
and up projections are one matrix, the experts of a layer are stacked, and every dimension is zero-padded to a multiple of
eight."""
from __future__ import annotations

import json
import math
import mmap
import os
import struct
from typing import Callable, Dict, List, Optional, Tuple

import torch

from ..config import HybridConfig, LatentAttentionConfig, MoEConfig, WindowAttentionConfig

_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64}


def round8(n: int) -> int:
    return (n + 7) // 8 * 8


class SafetensorsFile:
    """Memory-mapped reader: an 8-byte little-endian header length, a JSON header ``name -> dtype, shape, data_offsets``,
    then the data."""

    def __init__(self, path: str):
        self._f = open(path, "rb")
        size = os.fstat(self._f.fileno()).st_size
        n = struct.unpack("<Q", self._f.read(8))[0]
        if n > size - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
        self.header = json.loads(self._f.read(n))
        self.header.pop("__metadata__", None)
        self._base = 8 + n
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ) if size else None
        for name, e in self.header.items():
            lo, hi = e["data_offsets"]
            want = math.prod(e["shape"]) * torch.empty(0, dtype=_DTYPES[e["dtype"]]).element_size()
            if not 0 <= lo <= hi <= size - self._base or hi - lo != want:
                raise ValueError(f"{path}: {name} does not fit its shape or the file")

    def names(self) -> List[str]:
        return list(self.header)

    def __contains__(self, name: str) -> bool:
        return name in self.header

    def __getitem__(self, name: str) -> torch.Tensor:
        e = self.header[name]
        lo, hi = e["data_offsets"]
        raw = bytearray(self._map[self._base + lo:self._base + hi])
        if not raw:
            return torch.empty(e["shape"], dtype=_DTYPES[e["dtype"]])
        return torch.frombuffer(raw, dtype=_DTYPES[e["dtype"]]).view(e["shape"])


def write_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    inv = {v: k for k, v in _DTYPES.items()}
    header, off, blobs = {}, 0, []
    for name, t in tensors.items():
        b = t.detach().cpu().contiguous().view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": inv[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        off += len(b)
        blobs.append(b)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for b in blobs:
            f.write(b)


def hybrid_tensor_shapes(cfg: HybridConfig) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a checkpoint of this design."""
    d, out = cfg.d_model, {"embed": (cfg.vocab_size, cfg.d_model)}

    def feed_forward(p: str, ff: int, gated: bool) -> None:
        if gated:
            out[p + "gate"] = (ff, d)
        out.update({p + "up": (ff, d), p + "down": (d, ff)})

    if cfg.loop is not None:
        out.update({"loop.in": (d, 2 * d), "loop.step": (cfg.loop.times, d)})
    for i, layer in enumerate(cfg.layers):
        if cfg.owner(i) != i:
            continue
        p, m = f"l{i}.", layer.mixer
        H = m.heads
        out[p + "norm1"] = (d,)
        if isinstance(m, LatentAttentionConfig):
            out.update({p + "mix.q": (H * (m.dim + m.rot_dim), d), p + "mix.dkv": (m.kv_rank + m.rot_dim, d),
                        p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (H * m.dim, m.kv_rank),
                        p + "mix.uv": (H * m.vdim, m.kv_rank), p + "mix.sink": (H,), p + "mix.g": (H, d)})
        elif isinstance(m, WindowAttentionConfig):
            for n, rows in (("q", H * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                out.update({p + f"mix.{n}": (rows, d), p + f"mix.{n}.b": (rows,)})
            out.update({p + "mix.q.norm": (H * m.dim,), p + "mix.k.norm": (m.kv_heads * m.dim,), p + "mix.sink": (H,),
                        p + "mix.o.b": (d,)})
        else:
            for n, rows in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", H * m.vdim)):
                out[p + f"mix.{n}"] = (rows, d)
                out[p + f"mix.{n}.conv"] = (rows, m.conv)
            out.update({p + "mix.b": (H, d), p + "mix.a": (H, d), p + "mix.A_log": (H,), p + "mix.dt_bias": (H,),
                        p + "mix.norm": (m.vdim,), p + "mix.g": (H * m.vdim, d)})
        out[p + "mix.o"] = (d, H * m.vdim)
        if layer.mlp is not None:
            out[p + "norm2"] = (d,)
        if isinstance(layer.mlp, MoEConfig):
            for e in range(layer.mlp.experts):
                feed_forward(f"{p}mlp.e{e}.", layer.mlp.ff, True)
            out[p + "mlp.router"] = (layer.mlp.experts, d)
            if layer.mlp.shared_ff is not None:
                feed_forward(p + "mlp.shared.", layer.mlp.shared_ff, True)
        elif layer.mlp is not None:
            feed_forward(p + "mlp.", layer.mlp.ff, layer.mlp.gated)
    out["final.norm"] = (d,)
    out["head"] = (cfg.vocab_size, d)
    return out


def random_source(cfg: HybridConfig, device, seed: int = 0) -> Callable[[str], torch.Tensor]:
    """Random weights of the design's shapes (generated on ``device``, tensor by tensor)."""
    shapes = hybrid_tensor_shapes(cfg)
    number = {name: i for i, name in enumerate(shapes)}
    gen = torch.Generator(device=device)

    def get(name: str) -> torch.Tensor:
        shape = shapes[name]
        gen.manual_seed(seed * 100003 + number[name])
        t = torch.randn(*shape, device=device, generator=gen)
        if name.endswith((".conv",)) or (len(shape) == 2 and name not in ("embed", "loop.step")):
            t /= math.sqrt(shape[1])
        elif name.endswith((".dkv.norm", "mix.norm", ".q.norm", ".k.norm")):
            t = 1.0 + 0.1 * t
        elif name.endswith(("norm1", "norm2", "final.norm")):
            t = 1.0 - cfg.norm_gain_offset + 0.1 * t
        elif name.endswith("dt_bias"):
            t -= 2.0
        elif name != "embed":
            t *= 0.1
        return t.bfloat16()

    return get


class LayerWeights:
    """Packed tensors of one layer (see the module docstring)."""

    step_w: torch.Tensor                # [mixer input projections | up projection], one launch of a decode step
    in_w: torch.Tensor                  # the first part of it, zero rows up to a multiple of 16 included
    in_b: Optional[torch.Tensor] = None  # fp32 biases of the first part
    offs: Tuple[int, ...]               # first column of each projection in the product
    n_split: Optional[int] = None       # columns from here on leave in fp32 (decay and step-size projections)
    off_a: int = 0
    up_w: Optional[torch.Tensor] = None  # the second part
    out_w: torch.Tensor                 # [mixer output projection | feed-forward down projection]
    out_b: Optional[torch.Tensor] = None
    o_cols: int                         # columns of the mixer part (padded)
    mix: Dict[str, torch.Tensor]
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor] = None
    # layers whose feed-forward follows the mixer: [gate | up] and down, or the tensors of routed experts
    gu_w: Optional[torch.Tensor] = None
    down_w: Optional[torch.Tensor] = None
    moe: Optional[Dict[str, torch.Tensor]] = None


class HybridWeights:
    def __init__(self, cfg: HybridConfig, get: Callable[[str], torch.Tensor], dtype: torch.dtype, device):
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        self.shapes = hybrid_tensor_shapes(cfg)
        self._get = get
        self.d, self.dp = cfg.d_model, round8(cfg.d_model)
        self.embed = self._tensor("embed")
        self.head = self._rows([self._tensor("head")])[0]
        # a scale of the logits goes into the product's epilogue beside a bias of zeros
        self.head_b = self._bias([], self.head.shape[0]) if cfg.logit_scale != 1.0 else None
        self.final_norm = self._vec("final.norm")
        if cfg.loop is not None:
            w = self._tensor("loop.in")
            self.loop_w = torch.zeros(self.dp, 2 * self.dp, device=self.device, dtype=dtype)
            self.loop_w[:self.d, :self.d] = w[:, :self.d]
            self.loop_w[:self.d, self.dp:self.dp + self.d] = w[:, self.d:]
            self.loop_step = [self._bias([(0, t)], self.dp) for t in self._tensor("loop.step")]
        self.layers: Dict[int, LayerWeights] = {}
        for i, layer in enumerate(cfg.layers):
            if cfg.owner(i) == i:
                self.layers[i] = self._layer(i, layer)
        self._get = None

    # ------------------------------------------------------------------ pieces
    def _tensor(self, name: str) -> torch.Tensor:
        t = self._get(name)
        if tuple(t.shape) != tuple(self.shapes[name]):
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {tuple(self.shapes[name])}")
        return t.to(self.device, self.dtype)

    def _vec(self, name: str) -> torch.Tensor:
        t = self._tensor(name)
        out = torch.zeros(round8(t.numel()), device=self.device, dtype=self.dtype)
        out[:t.numel()] = t
        return out

    def _rows(self, parts, align=None) -> Tuple[torch.Tensor, Tuple[int, ...]]:
        """Stack matrices with the same columns; part j starts at a multiple of ``align[j]`` (8) rows."""
        offs, n = [], 0
        for j, t in enumerate(parts):
            a = 8 if align is None else align[j]
            n = (n + a - 1) // a * a
            offs.append(n)
            n += t.shape[0]
        out = torch.zeros(round8(n), round8(parts[0].shape[1]), device=self.device, dtype=self.dtype)
        for o, t in zip(offs, parts):
            out[o:o + t.shape[0], :t.shape[1]] = t
        return out, tuple(offs)

    def _bias(self, parts, n: int) -> torch.Tensor:
        """fp32 vector of ``n`` entries, up to a multiple of 32 of zeros: the vectors of ``parts`` at their offsets."""
        out = torch.zeros((n + 31) // 32 * 32, device=self.device, dtype=torch.float32)
        for o, t in parts:
            out[o:o + t.numel()] = t.float()
        return out

    def _gate_up(self, p: str) -> torch.Tensor:
        """``(2 F, dp)``: gate rows, then up rows, each padded to a multiple of eight."""
        g, u = self._tensor(p + "gate"), self._tensor(p + "up")
        out = torch.zeros(2, round8(g.shape[0]), self.dp, device=self.device, dtype=self.dtype)
        out[0, :g.shape[0], :self.d], out[1, :g.shape[0], :self.d] = g, u
        return out.view(-1, self.dp)

    def _down(self, p: str) -> torch.Tensor:
        return self._rows([self._tensor(p + "down")])[0]

    def _experts(self, p: str, f: MoEConfig) -> Dict[str, torch.Tensor]:
        F, kw = round8(f.ff), dict(device=self.device, dtype=self.dtype)
        out = {"router": self._rows([self._tensor(p + "router")])[0], "gu": torch.empty(f.experts, 2 * F, self.dp, **kw),
               "down": torch.empty(f.experts, self.dp, F, **kw)}
        for e in range(f.experts):
            out["gu"][e], out["down"][e] = self._gate_up(f"{p}e{e}."), self._down(f"{p}e{e}.")
        if f.shared_ff is not None:
            out["sh_gu"], out["sh_down"] = self._gate_up(p + "shared."), self._down(p + "shared.")
        return out

    def _layer(self, i: int, layer) -> LayerWeights:
        p, m, L = f"l{i}.", layer.mixer, LayerWeights()
        t = lambda n: self._tensor(p + "mix." + n)
        L.norm1 = self._vec(p + "norm1")
        if isinstance(m, WindowAttentionConfig):
            parts = ("q", "k", "v")
            L.in_w, L.offs = self._rows([t(n) for n in parts])
            L.in_b = self._bias([(o, t(n + ".b")) for o, n in zip(L.offs, parts)], L.in_w.shape[0])
            L.out_b = self._bias([(0, t("o.b"))], self.dp)
            inv = torch.tensor(m.rot.inv_freq(), dtype=torch.float64).to(self.device, torch.float32)
            L.mix = {"q_norm": t("q.norm").contiguous(), "k_norm": t("k.norm").contiguous(), "inv_freq": inv,
                     "sink": t("sink").float().contiguous()}
        elif isinstance(m, LatentAttentionConfig):
            L.in_w, L.offs = self._rows([t("q"), t("dkv"), t("g")])
            uk, uv = t("uk"), t("uv")
            w, (ok, ov) = self._rows([uk, uv])
            inv = torch.tensor(m.rot.inv_freq(), dtype=torch.float64).to(self.device, torch.float32)
            L.mix = {"c_norm": t("dkv.norm").contiguous(), "inv_freq": inv, "ukv": w, "uk": w[ok:ok + uk.shape[0]],
                     "uv": w[ov:ov + uv.shape[0]], "uv_off": ov, "sink": t("sink").float().contiguous()}
        else:
            parts = [t("q"), t("k"), t("v"), t("g"), t("b"), t("a")]
            L.in_w, offs = self._rows(parts, align=[8, 8, 8, 8, 32, 8])
            L.offs, L.n_split, L.off_a = offs[:4], offs[4], offs[5] - offs[4]
            L.mix = {"conv_q": t("q.conv").contiguous(), "conv_k": t("k.conv").contiguous(),
                     "conv_v": t("v.conv").contiguous(), "a_log": t("A_log").contiguous(),
                     "dt_bias": t("dt_bias").contiguous(), "norm": t("norm").contiguous()}
        o = t("o")
        L.o_cols = round8(o.shape[1])
        f = layer.mlp
        ff = f.ff if f is not None and self.cfg.design.parallel else 0
        L.out_w = torch.zeros(self.dp, L.o_cols + round8(ff), device=self.device, dtype=self.dtype)
        L.out_w[:self.d, :o.shape[1]] = o
        L.step_w = L.in_w
        if f is None:
            return L
        L.norm2 = self._vec(p + "norm2")
        if self.cfg.design.parallel:
            L.step_w, (_, up) = self._rows([L.in_w[:, :self.d], self._tensor(p + "mlp.up")], align=[8, 16])
            L.in_w, L.up_w = L.step_w[:up], L.step_w[up:]
            L.out_w[:self.d, L.o_cols:L.o_cols + ff] = self._tensor(p + "mlp.down")
        elif isinstance(f, MoEConfig):
            L.moe = self._experts(p + "mlp.", f)
        else:
            L.gu_w, L.down_w = self._gate_up(p + "mlp."), self._down(p + "mlp.")
        return L

    def bytes(self) -> int:
        n = self.embed.numel() + self.head.numel()
        for L in self.layers.values():
            n += L.step_w.numel() + L.out_w.numel()
            n += L.mix["ukv"].numel() if "ukv" in L.mix else 0
            n += sum(t.numel() for t in (L.gu_w, L.down_w, *(L.moe or {}).values()) if t is not None)
        return n * self.embed.element_size()
