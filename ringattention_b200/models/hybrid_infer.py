"""Inference engine of hybrid decoders: every layer of the configuration names its mixer (latent attention over a cache of
latents, or the gated delta rule over a recurrent state), and the engine keeps what each needs between steps.

A layer adds its mixer and its feed-forward to the residual stream together, both computed from the same rows through
norms of their own: ``x += mixer(norm1(x)) + ff(norm2(x))``. One norm launch writes both normalised copies; the mixer
writes its heads and the up projection its activations side by side into one buffer, and one product with
``[W_o | W_down]`` adds both to the 32-bit residual stream.

Steps may cut the prompt anywhere: a step runs the tokens it brings from what earlier steps left. ``dtype`` bf16 is the
serving form (bf16 products with fp32 accumulation; norms, positions, scores, softmax, recurrences and the residual
stream in fp32); fp32 runs the same step functions with every product in true 32-bit."""
from __future__ import annotations

from typing import Callable, List, Optional, Sequence

import torch

from ..config import GatedDeltaConfig, HybridConfig, LatentAttentionConfig
from ..ops import kernels as K
from ..ops import mixers as X
from .cache import DeltaState, LatentCache
from .engine import InferenceEngine
from .weights import HybridWeights, random_source


class HybridInference(InferenceEngine):
    def __init__(self, cfg: HybridConfig, max_context: int, batch: int = 1, device="cuda", seed: int = 0,
                 dtype: torch.dtype = torch.bfloat16, source: Optional[Callable[[str], torch.Tensor]] = None,
                 weights: Optional[HybridWeights] = None):
        """``source``: tensor name -> tensor of a checkpoint (random weights from ``seed`` when absent)."""
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("dtype must be bfloat16 or float32")
        super().__init__(batch, device, batch)
        self.cfg, self.dtype = cfg, dtype
        self.S_max = max_context
        self.W = weights if weights is not None else HybridWeights(
            cfg, source if source is not None else random_source(cfg, self.device, seed), dtype, self.device)
        self.caches = [LatentCache(l.mixer, batch, max_context, self.device, dtype)
                       if isinstance(l.mixer, LatentAttentionConfig) else DeltaState(l.mixer, batch, self.device)
                       for l in cfg.layers]

    def cache_bytes(self) -> int:
        return sum(c.bytes() for c in self.caches)

    def _clear_cache(self) -> None:
        for c in self.caches:
            c.clear()

    def _check_room(self, n: int) -> None:
        if self.length + n > self.S_max:
            raise ValueError("context exceeds max_context")

    # ------------------------------------------------------------------ one layer
    def _mixer(self, i: int, L, proj, tail, out, T: int, n_rows: int) -> None:
        m, c, eps = self.cfg.layers[i].mixer, self.caches[i], self.cfg.rms_eps
        if isinstance(m, GatedDeltaConfig):
            X.delta_mixer(proj, tail, out, B=self.B, T=T, m=m, offs=L.offs, off_a=L.off_a, w=L.mix, ring=c.ring,
                          state=c.state, eps=eps, pos=self.state)
        else:
            X.latent_mixer(proj, out, B=self.B, T=T, m=m, offs=L.offs, w=L.mix, cache=c.data, n_rows=n_rows, eps=eps,
                           pos=self.state)

    def _layer(self, i: int, x: torch.Tensor, T: int, n_rows: int) -> None:
        cfg, W = self.cfg, self.W
        layer, L = cfg.layers[i], W.layers[cfg.owner(i)]
        rows, dev = x.shape[0], self.device
        h1, h2 = K.norm_f32(x, W.d, cfg.rms_eps, cfg.norm_gain_offset, L.norm1, L.norm2)
        n = L.in_w.shape[0]
        main = n if L.n_split is None else L.n_split
        proj = torch.empty(rows, main, device=dev, dtype=self.dtype)
        tail = None if main == n else torch.empty(rows, n - main, device=dev, dtype=torch.float32)
        both = torch.empty(rows, L.out_w.shape[1], device=dev, dtype=self.dtype)  # [heads | activations]
        acts = both[:, L.o_cols:] if L.up_w is not None else None
        few = rows <= 8 and self.dtype == torch.bfloat16
        if few:  # every projection of the layer's input in one launch
            K.linear_segments(h1, L.step_w, x2=h2, y=proj, y32=tail, ya=acts, n32_from=L.n_split,
                              act_from=None if acts is None else L.step_w.shape[0] - L.up_w.shape[0])
        else:
            K.linear_ex(h1, L.in_w, proj, tail=tail, n_split=L.n_split)
        o_real = layer.mixer.heads * layer.mixer.vdim
        if o_real != L.o_cols:
            both[:, o_real:L.o_cols].zero_()
        self._mixer(i, L, proj, tail, both[:, :o_real], T, n_rows)
        if acts is not None and not few:
            K.linear_ex(h2, L.up_w, acts, relu2=True)
        K.linear_ex(both, L.out_w, x, residual=x)

    def _forward(self, tokens: torch.Tensor, T: int, n_rows: int, rows_idx: Optional[torch.Tensor],
                 taps: Optional[List[torch.Tensor]] = None) -> Optional[torch.Tensor]:
        """``tokens (B*T,)`` int32 at positions ``state[0] ..``; logits of the rows in ``rows_idx`` (None: all)."""
        cfg, W = self.cfg, self.W
        x = torch.empty(tokens.numel(), W.dp, device=self.device, dtype=torch.float32)
        K.embed_f32(tokens, W.embed, W.d, x)
        for i in range(cfg.n_layers):
            self._layer(i, x, T, n_rows)
            if taps is not None:
                taps.append(x[:, :W.d].clone())
        if rows_idx is not None and rows_idx.numel() == 0:
            return None
        hf, _ = K.norm_f32(x, W.d, cfg.rms_eps, cfg.norm_gain_offset, W.final_norm, rows_idx=rows_idx)
        logits = torch.empty(hf.shape[0], W.head.shape[0], device=self.device, dtype=torch.float32)
        K.linear_ex(hf, W.head, logits)
        return logits[:, :cfg.vocab_size]

    # ------------------------------------------------------------------ steps
    @torch.no_grad()
    def step(self, tokens: torch.Tensor, want: Optional[Sequence[int]] = None,
             taps: Optional[List[torch.Tensor]] = None) -> Optional[torch.Tensor]:
        """Append ``tokens (B, T)`` to every sequence. ``want``: places among these tokens whose logits are returned,
        ``(B, len(want), vocab)`` fp32 (all of them when None; None is returned for an empty list)."""
        B, T = tokens.shape
        if B != self.B or T < 1:
            raise ValueError(f"step takes ({self.B}, T >= 1) tokens")
        self._check_room(T)
        self.state[0] = self.length
        idx = None
        if want is not None:
            if any(not 0 <= w < T for w in want):
                raise ValueError("want names a place outside the step")
            idx = torch.tensor([b * T + w for b in range(B) for w in want], dtype=torch.int32, device=self.device)
        flat = tokens.to(self.device, torch.int32).reshape(-1).contiguous()
        logits = self._forward(flat, T, self.length + T, idx, taps)
        self.length += T
        return None if logits is None else logits.view(B, -1, self.cfg.vocab_size)

    @torch.no_grad()
    def prefill_chunk(self, tokens: torch.Tensor) -> torch.Tensor:
        return self.step(tokens, want=[tokens.shape[1] - 1])[:, 0]

    def _decode_body(self, tokens: torch.Tensor) -> torch.Tensor:
        logits = self._forward(tokens, 1, self.S_max, None)
        K.decode_advance(self.state)
        return logits
