"""What a sequence leaves behind between steps: caches that grow by one row per token and recurrent states of fixed size.

An engine holds one object per layer (layers that share weights still have one each). ``bytes()`` is what it occupies,
``clear()`` forgets the sequences; the memory stays."""
from __future__ import annotations

import torch

from ..config import GatedDeltaConfig, LatentAttentionConfig, WindowAttentionConfig


class KVCache:
    """Keys and values per head. Heads-major storage ``(B, 2, H, S_max, D)``: the rows of one (k|v, head) are contiguous,
    so every CTA of the split-KV decode kernel streams one long run instead of 256-byte pieces 16 KB apart. The kernels
    see ``(B, S_max, H, D)`` views with strides; the flash kernel's tensor maps and the decode kernel take any strides."""

    def __init__(self, batch: int, heads: int, rows: int, dim: int, device, dtype=torch.bfloat16):
        self.data = torch.zeros(batch, 2, heads, rows, dim, device=device, dtype=dtype)
        self.k = self.data[:, 0].permute(0, 2, 1, 3)
        self.v = self.data[:, 1].permute(0, 2, 1, 3)

    def bytes(self) -> int:
        return self.data.numel() * self.data.element_size()

    def clear(self) -> None:
        """Rows past the engine's row count are never read: nothing to do."""


class LatentCache:
    """One row ``[latent | shared rotated key]`` per token, both parts padded to multiples of eight elements."""

    def __init__(self, m: LatentAttentionConfig, batch: int, rows: int, device, dtype):
        width = (m.kv_rank + 7) // 8 * 8 + (m.rot_dim + 7) // 8 * 8
        self.data = torch.zeros(batch, rows, width, device=device, dtype=dtype)

    def bytes(self) -> int:
        return self.data.numel() * self.data.element_size()

    def clear(self) -> None:
        """Rows past the engine's length are never read: nothing to do."""


class WindowCache:
    """Keys and values of the last tokens in a ring per head: position p in row ``p % rows``, heads-major ``(B, G, rows, dim)``
    with dims padded to multiples of eight. ``rows`` is a multiple of 128 (key tiles never straddle the end of the ring) that
    holds the windows of all tokens of a step of ``max_step`` tokens, or the whole context where that is less."""

    def __init__(self, m: WindowAttentionConfig, batch: int, context: int, max_step: int, device, dtype):
        self.window = context if m.window is None else min(m.window, context)
        whole, ring = (context + 127) // 128 * 128, (self.window - 1 + max_step + 127 + 127) // 128 * 128
        self.rows = min(whole, ring)
        pad = lambda n: (n + 7) // 8 * 8
        self.k = torch.zeros(batch, m.kv_heads, self.rows, pad(m.dim), device=device, dtype=dtype)
        self.v = torch.zeros(batch, m.kv_heads, self.rows, pad(m.vdim), device=device, dtype=dtype)

    def bytes(self) -> int:
        return (self.k.numel() + self.v.numel()) * self.k.element_size()

    def clear(self) -> None:
        """Rows of positions past the engine's length are never read: nothing to do."""


class DeltaState:
    """Recurrent state of the gated delta rule (transposed, ``(B, H, dv, dk)``) and the ring of the last ``conv`` inputs of
    its short convolutions (position p in row ``p % conv``); 32-bit."""

    def __init__(self, m: GatedDeltaConfig, batch: int, device):
        self.state = torch.zeros(batch, m.heads, m.vdim, m.dim, device=device, dtype=torch.float32)
        self.ring = torch.zeros(batch, m.conv, 2 * m.kv_heads * m.dim + m.heads * m.vdim, device=device,
                                dtype=torch.float32)

    def bytes(self) -> int:
        return 4 * (self.state.numel() + self.ring.numel())

    def clear(self) -> None:
        self.state.zero_()
        self.ring.zero_()
