"""Inference engine of hybrid decoders: every layer of the configuration names its mixer (latent attention over a cache of
latents, the gated delta rule over a recurrent state, attention over a ring of the last keys and values) and its feed-forward
(dense, gated, routed experts), and the engine keeps what each layer run needs between steps.

Layers are added to the residual stream in one of two ways. In parallel, ``x += mixer(norm1(x)) + ff(norm2(x))``: one norm
launch writes both normalised copies; the mixer writes its heads and the up projection its activations side by side into one
buffer, and one product with ``[W_o | W_down]`` adds both to the 32-bit residual stream. In sequence,
``x += mixer(norm1(x))``, then ``x += ff(norm2(x))``. Layers of a loop run several times with the same tensors; a pass
begins with a product over the stream and the embedding side by side.

Steps may cut the prompt anywhere: a step runs the tokens it brings from what earlier steps left. ``dtype`` bf16 is the
serving form (bf16 products with fp32 accumulation; norms, positions, scores, softmax, routers, recurrences and the residual
stream in fp32); fp32 runs the same step functions with every product in true 32-bit."""
from __future__ import annotations

from typing import Callable, List, Optional, Sequence

import torch

from ..config import GatedDeltaConfig, HybridConfig, LatentAttentionConfig, WindowAttentionConfig
from ..ops import experts as E
from ..ops import kernels as K
from ..ops import mixers as X
from .cache import DeltaState, LatentCache, WindowCache
from .engine import InferenceEngine
from .weights import HybridWeights, random_source


class HybridInference(InferenceEngine):
    def __init__(self, cfg: HybridConfig, max_context: int, batch: int = 1, device="cuda", seed: int = 0,
                 dtype: torch.dtype = torch.bfloat16, source: Optional[Callable[[str], torch.Tensor]] = None,
                 weights: Optional[HybridWeights] = None, max_step: int = 8192):
        """``source``: tensor name -> tensor of a checkpoint (random weights from ``seed`` when absent). ``max_step``: tokens
        of a sequence that run at once where a layer keeps a window only (longer steps are cut); it sizes the windows' rings."""
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("dtype must be bfloat16 or float32")
        super().__init__(batch, device, batch)
        self.cfg, self.dtype = cfg, dtype
        self.S_max = max_context
        self.W = weights if weights is not None else HybridWeights(
            cfg, source if source is not None else random_source(cfg, self.device, seed), dtype, self.device)
        self.max_step = max_step
        self.runs = cfg.runs
        self.caches = [self._make_cache(cfg.layers[r.layer].mixer) for r in self.runs]
        self.cut = any(isinstance(c, WindowCache) for c in self.caches)

    def _make_cache(self, m):
        if isinstance(m, LatentAttentionConfig):
            return LatentCache(m, self.B, self.S_max, self.device, self.dtype)
        if isinstance(m, WindowAttentionConfig):
            return WindowCache(m, self.B, self.S_max, self.max_step, self.device, self.dtype)
        return DeltaState(m, self.B, self.device)

    def cache_bytes(self) -> int:
        return sum(c.bytes() for c in self.caches)

    def _clear_cache(self) -> None:
        for c in self.caches:
            c.clear()

    def _check_room(self, n: int) -> None:
        if self.length + n > self.S_max:
            raise ValueError("context exceeds max_context")

    # ------------------------------------------------------------------ one layer
    def _mixer(self, run: int, L, proj, tail, out, T: int, length: int, n_rows: int) -> None:
        m, c, eps = self.cfg.layers[self.runs[run].layer].mixer, self.caches[run], self.cfg.rms_eps
        if isinstance(m, GatedDeltaConfig):
            X.delta_mixer(proj, tail, out, B=self.B, T=T, m=m, offs=L.offs, off_a=L.off_a, w=L.mix, ring=c.ring,
                          state=c.state, eps=eps, pos=self.state)
        elif isinstance(m, WindowAttentionConfig):
            X.window_mixer(proj, out, B=self.B, T=T, m=m, offs=L.offs, w=L.mix, cache=c, length=length, eps=eps,
                           pos=self.state)
        else:
            X.latent_mixer(proj, out, B=self.B, T=T, m=m, offs=L.offs, w=L.mix, cache=c.data, n_rows=n_rows, eps=eps,
                           pos=self.state)

    def _parallel_layer(self, run: int, x: torch.Tensor, T: int, length: int, n_rows: int) -> None:
        cfg, W = self.cfg, self.W
        i = self.runs[run].layer
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
        self._mixer(run, L, proj, tail, both[:, :o_real], T, length, n_rows)
        if acts is not None and not few:
            K.linear_ex(h2, L.up_w, acts, relu2=True)
        K.linear_ex(both, L.out_w, x, residual=x)

    def _sequential_layer(self, run: int, x: torch.Tensor, T: int, length: int, n_rows: int) -> None:
        cfg, W = self.cfg, self.W
        i = self.runs[run].layer
        layer, L = cfg.layers[i], W.layers[cfg.owner(i)]
        new = lambda n: torch.empty(x.shape[0], n, device=self.device, dtype=self.dtype)
        h, _ = K.norm_f32(x, W.d, cfg.rms_eps, cfg.norm_gain_offset, L.norm1)
        proj, heads = new(L.in_w.shape[0]), new(L.o_cols)
        K.linear_ex(h, L.in_w, proj, bias=L.in_b)
        o_real = layer.mixer.heads * layer.mixer.vdim
        if o_real != L.o_cols:
            heads[:, o_real:].zero_()
        self._mixer(run, L, proj, None, heads[:, :o_real], T, length, n_rows)
        K.linear_ex(heads, L.out_w, x, residual=x, bias=L.out_b)
        if layer.mlp is None:
            return
        h, _ = K.norm_f32(x, W.d, cfg.rms_eps, cfg.norm_gain_offset, L.norm2)
        if L.moe is not None:
            E.moe_(x, h, W.d, layer.mlp, L.moe)
        else:
            hidden = new(L.down_w.shape[1])
            K.linear_gated(h, L.gu_w, hidden)
            K.linear_ex(hidden, L.down_w, x, residual=x)

    def _enter_pass(self, t: int, tokens: torch.Tensor, x: torch.Tensor) -> None:
        K.linear_ex(K.stream_pair(tokens, self.W.embed, x, self.W.d), self.W.loop_w, x, bias=self.W.loop_step[t])

    def _forward(self, tokens: torch.Tensor, T: int, length: int, n_rows: int, rows_idx: Optional[torch.Tensor],
                 taps: Optional[List[torch.Tensor]] = None) -> Optional[torch.Tensor]:
        """``tokens (B*T,)`` int32 at positions ``state[0] ..``; logits of the rows in ``rows_idx`` (None: all). ``length``:
        tokens before them, ``n_rows``: tokens after the step (upper bounds in a step that is replayed)."""
        cfg, W = self.cfg, self.W
        x = torch.empty(tokens.numel(), W.dp, device=self.device, dtype=torch.float32)
        K.embed_f32(tokens, W.embed, W.d, x)
        layer = self._parallel_layer if cfg.design.parallel else self._sequential_layer
        for n, r in enumerate(self.runs):
            if r.enter is not None:
                self._enter_pass(r.enter, tokens, x)
            layer(n, x, T, length, n_rows)
            if taps is not None:
                taps.append(x[:, :W.d].clone())
        if rows_idx is not None and rows_idx.numel() == 0:
            return None
        hf, _ = K.norm_f32(x, W.d, cfg.rms_eps, cfg.norm_gain_offset, W.final_norm, rows_idx=rows_idx)
        logits = torch.empty(hf.shape[0], W.head.shape[0], device=self.device, dtype=torch.float32)
        K.linear_ex(hf, W.head, logits, bias=W.head_b, alpha=cfg.logit_scale)
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
        if want is not None and any(not 0 <= w < T for w in want):
            raise ValueError("want names a place outside the step")
        if self.cut and T > self.max_step:
            return self._long_step(tokens, want, taps)
        self.state[0] = self.length
        idx = None
        if want is not None:
            idx = torch.tensor([b * T + w for b in range(B) for w in want], dtype=torch.int32, device=self.device)
        flat = tokens.to(self.device, torch.int32).reshape(-1).contiguous()
        logits = self._forward(flat, T, self.length, self.length + T, idx, taps)
        self.length += T
        return None if logits is None else logits.view(B, -1, self.cfg.vocab_size)

    def _long_step(self, tokens: torch.Tensor, want: Optional[Sequence[int]], taps) -> Optional[torch.Tensor]:
        """A step that is cut into portions of ``max_step`` tokens."""
        if taps is not None:
            raise ValueError("a step that is cut has no taps")
        out, places, T = [], [], tokens.shape[1]
        for c0 in range(0, T, self.max_step):
            n = min(self.max_step, T - c0)
            here = list(range(T)) if want is None else [w for w in want if c0 <= w < c0 + n]
            here = [w for w in here if c0 <= w < c0 + n]
            got = self.step(tokens[:, c0:c0 + n], want=[w - c0 for w in here])
            if got is not None:
                out.append(got)
                places += here
        if not out:
            return None
        order = list(range(T)) if want is None else list(want)
        first = {w: i for i, w in reversed(list(enumerate(places)))}
        return torch.cat(out, dim=1)[:, [first[w] for w in order]]

    @torch.no_grad()
    def prefill_chunk(self, tokens: torch.Tensor) -> torch.Tensor:
        return self.step(tokens, want=[tokens.shape[1] - 1])[:, 0]

    def _decode_body(self, tokens: torch.Tensor) -> torch.Tensor:
        logits = self._forward(tokens, 1, self.S_max, self.S_max, None)
        K.decode_advance(self.state)
        return logits
