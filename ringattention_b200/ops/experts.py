"""Routed experts (``moe.cu``, ``moe_gemm_sm100.cu``): sigmoid scores, the largest ``top`` of them, gated feed-forwards on the
input times the score, and a shared expert."""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from . import kernels as K

c_ll = ctypes.c_longlong
c_vp = ctypes.c_void_p
c_i = ctypes.c_int


class _MoeParams(ctypes.Structure):
    _fields_ = [("rows", c_i), ("d", c_i), ("dp", c_i), ("E", c_i), ("top", c_i), ("F", c_i), ("Fs", c_i),
                ("h", c_vp), ("logits", c_vp), ("ld_logits", c_ll), ("gu", c_vp), ("down", c_vp), ("sh_gu", c_vp),
                ("sh_down", c_vp), ("ids", c_vp), ("weight", c_vp), ("act", c_vp), ("x", c_vp), ("ldx", c_ll),
                ("count", c_vp), ("list", c_vp), ("y", c_vp), ("status", c_vp)]


def moe_(x, h, d: int, m, w) -> None:
    """``x += experts(h)``: ``x (rows, dp)`` the fp32 residual stream, ``h (rows, dp)`` its normed rows (bf16 or fp32).

    ``w``: ``router (E padded to 8, dp)``, ``gu (E, 2 F, dp)`` with gate rows before up rows, ``down (E, dp, F)``, and with a
    shared expert ``sh_gu (2 Fs, dp)``, ``sh_down (dp, Fs)``; all in ``h``'s type, widths padded to multiples of eight.
    ``m``: a :class:`~ringattention_b200.config.MoEConfig`. At most eight rows (and fp32) stream the weights of the experts
    that a token uses; more rows run as a grouped product over all experts."""
    rows, dp = h.shape
    dev, f32 = h.device, h.dtype == torch.float32
    F, Fs = w["down"].shape[2], 0 if m.shared_ff is None else w["sh_down"].shape[1]
    assert h.is_contiguous() and x.dtype == torch.float32 and x.stride(1) == 1 and x.shape == (rows, dp)
    assert w["gu"].shape == (m.experts, 2 * F, dp) and w["down"].shape == (m.experts, dp, F)
    logits = torch.empty(rows, w["router"].shape[0], device=dev, dtype=torch.float32)
    K.linear_ex(h, w["router"], logits)
    p = lambda t: t.data_ptr()
    weight = torch.empty(rows, m.top, device=dev, dtype=torch.float32)
    a = _MoeParams()
    a.rows, a.d, a.dp, a.E, a.top, a.F, a.Fs = rows, d, dp, m.experts, m.top, F, Fs
    a.h, a.logits, a.ld_logits, a.gu, a.down = p(h), p(logits), logits.stride(0), p(w["gu"]), p(w["down"])
    a.x, a.ldx, a.weight, a.status = p(x), x.stride(0), p(weight), p(_lib.status_tensor(dev))
    if f32 or rows <= 8:
        if Fs:
            a.sh_gu, a.sh_down = p(w["sh_gu"]), p(w["sh_down"])
        ids = torch.empty(rows, m.top, device=dev, dtype=torch.int32)
        act = torch.empty(rows, m.top * F + Fs, device=dev, dtype=h.dtype)
        a.ids, a.act = p(ids), p(act)
        return _lib.call("ra_moe_few", ctypes.byref(a), int(f32), _lib.stream_ptr(), n_kernels=2)
    count = torch.zeros(m.experts, device=dev, dtype=torch.int32)
    lists = torch.empty(m.experts, rows, device=dev, dtype=torch.int32)
    n = rows * m.top
    act = torch.empty(128 * (n // 128 + min(n, m.experts)), F, device=dev, dtype=h.dtype)  # row tiles expert by expert
    y = torch.empty(rows * m.top, dp, device=dev, dtype=h.dtype)
    a.count, a.list, a.act, a.y = p(count), p(lists), p(act), p(y)
    _lib.call("ra_moe_route", ctypes.byref(a), _lib.stream_ptr())
    _lib.call("ra_moe_gemm", ctypes.byref(a), _lib.stream_ptr(), n_kernels=2)
    _lib.call("ra_moe_combine", ctypes.byref(a), _lib.stream_ptr())
    if Fs:
        hidden = torch.empty(rows, Fs, device=dev, dtype=h.dtype)
        K.linear_gated(h, w["sh_gu"], hidden)
        K.linear_ex(hidden, w["sh_down"], x, residual=x)
