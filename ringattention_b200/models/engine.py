"""The serving loop shared by the inference engines: chunked prefill, decoding one token per sequence and step (eagerly or
as one replayed CUDA graph), greedy sampling, and the step counters on the device that make a decode step replayable.

An engine supplies ``prefill_chunk`` (append a chunk, return the last position's logits), ``_decode_body`` (all launches of
one decode step, every per-token scalar read from ``state``) and ``_clear_cache``."""
from __future__ import annotations

import time
from typing import List

import torch


class InferenceEngine:
    def __init__(self, batch: int, device, token_rows: int):
        self.device = torch.device(device)
        self.B = batch
        self.length = 0                             # tokens in the cache (global)
        # [position, step] on the device: lets one recorded CUDA graph serve every decode step
        self.state = torch.zeros(2, dtype=torch.int64, device=self.device)
        self._graph = None
        self._tok_buf = torch.zeros(token_rows, dtype=torch.int32, device=self.device)

    # ------------------------------------------------------------------ supplied by the engine
    def prefill_chunk(self, tokens: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def _decode_body(self, tokens: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def _clear_cache(self) -> None:
        raise NotImplementedError

    def _check_room(self, n: int) -> None:
        """Raise when ``n`` more tokens do not fit (engines with a fixed cache size override it)."""

    def first_tokens(self, logits: torch.Tensor) -> torch.Tensor:
        """The tokens decoding starts with, from the prompt's last logits."""
        return self.sample(logits)

    # ------------------------------------------------------------------ sampling
    @staticmethod
    def sample(logits: torch.Tensor) -> torch.Tensor:
        """Greedy."""
        return logits.argmax(dim=-1)

    # ------------------------------------------------------------------ decode
    @torch.no_grad()
    def decode_step(self, tokens: torch.Tensor) -> torch.Tensor:
        """One token per sequence: ``tokens (B,)`` -> logits ``(B, vocab)`` fp32 (same on all ranks)."""
        self._check_room(1)
        self.state[0] = self.length
        logits = self._decode_body(tokens.to(self.device, torch.int32).reshape(-1).contiguous())
        self.length += 1
        return logits

    @torch.no_grad()
    def decode_step_graph(self) -> torch.Tensor:
        """Greedy step on the token in ``self._tok_buf`` through a CUDA graph recorded on first use:
        one replay per token instead of a handful of launches per layer. Writes the next token back into
        ``self._tok_buf`` and returns it. Call :meth:`decode_step` at least once before (buffers and
        kernels must exist before capture)."""
        self._check_room(1)
        if self._graph is None:
            self.state[0] = self.length
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g):
                logits = self._decode_body(self._tok_buf)
                self._tok_buf.copy_(self.sample(logits).to(torch.int32))
            self._graph = g
        self._graph.replay()
        self.length += 1
        return self._tok_buf

    def reset(self) -> None:
        """Forget the cached context (the cache memory is kept). The recorded decode graph is dropped
        too: it may hold properties of the prefilled context as launch constants."""
        self.length = 0
        self.state.zero_()
        self._graph = None
        self._clear_cache()

    # ------------------------------------------------------------------ generation
    @torch.no_grad()
    def generate(self, prompt: torch.Tensor, new_tokens: int, chunk: int = 32768, use_graph: bool = True):
        """Chunked prefill of ``prompt (B, T)`` followed by greedy decoding. Returns the generated
        tokens ``(B, new_tokens)`` and timing: prefill seconds, per-token decode latencies."""
        B, T = prompt.shape
        if self.length:
            self.reset()
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        logits = None
        for c0 in range(0, T, chunk):
            logits = self.prefill_chunk(prompt[:, c0:c0 + chunk])
        torch.cuda.synchronize()
        t_prefill = time.perf_counter() - t0
        out: List[torch.Tensor] = []
        lat: List[float] = []
        nxt = self.first_tokens(logits)
        for i in range(new_tokens):
            out.append(nxt.clone())
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            if use_graph and i >= 2:
                if i == 2:
                    self._tok_buf.copy_(nxt.to(torch.int32))
                nxt = self.decode_step_graph()
            else:
                nxt = self.sample(self.decode_step(nxt))
            e1.record()
            torch.cuda.synchronize()
            lat.append(e0.elapsed_time(e1))
        return torch.stack([t.to(torch.int64) for t in out], dim=1), {"prefill_s": t_prefill, "decode_ms": lat}
