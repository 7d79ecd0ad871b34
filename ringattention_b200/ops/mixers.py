"""Bindings of the token mixers of hybrid decoders: the gated delta rule (``delta_sm100.cu``) and latent attention
(``latent_sm100.cu``). Activations and weights are bf16 or fp32 throughout (one type per call); states, decays, scores
and softmax are fp32 in both."""
from __future__ import annotations

import ctypes

import torch

from . import _lib

c_ll = ctypes.c_longlong
c_vp = ctypes.c_void_p
c_i = ctypes.c_int
c_f = ctypes.c_float


def _p(t) -> int:
    return 0 if t is None else t.data_ptr()


class _DeltaParams(ctypes.Structure):
    _fields_ = [("B", c_i), ("T", c_i), ("H", c_i), ("G", c_i), ("dk", c_i), ("dv", c_i), ("taps", c_i),
                ("proj", c_vp), ("ldp", c_ll),
                ("off_q", c_i), ("off_k", c_i), ("off_v", c_i), ("off_g", c_i),
                ("ba", c_vp), ("ldba", c_ll), ("off_a", c_i),
                ("conv_q", c_vp), ("conv_k", c_vp), ("conv_v", c_vp),
                ("a_log", c_vp), ("dt_bias", c_vp), ("norm_w", c_vp),
                ("ring", c_vp), ("state", c_vp),
                ("q", c_vp), ("k", c_vp), ("v", c_vp), ("gb", c_vp), ("o", c_vp),
                ("out", c_vp), ("ldo", c_ll), ("eps", c_f), ("q_scale", c_f), ("pos", c_vp)]


def delta_mixer(proj, ba, out, *, B: int, T: int, m, offs, off_a: int, w, ring, state, eps: float, pos) -> None:
    """Gated delta rule over ``T`` new tokens of each of ``B`` sequences.

    ``proj (B*T, ld)``: projections with q, k, v and the gate at columns ``offs``; ``ba (B*T, ld)`` fp32: the step-size
    projection and, from ``off_a``, the decay projection. ``w``: ``conv_q/k/v``, ``a_log``, ``dt_bias``, ``norm`` in
    ``proj``'s type. ``ring (B, taps, channels)`` and ``state (B, H, dv, dk)`` fp32 are updated in place. ``out (B*T, >=
    H*dv)``: a row-strided view. ``m``: a :class:`~ringattention_b200.config.GatedDeltaConfig`; ``pos``: int64 on the
    device, the position of the first new token."""
    dev = proj.device
    rows, H, G, dk, dv = B * T, m.heads, m.kv_heads, m.dim, m.vdim
    assert proj.shape[0] == rows and proj.stride(1) == 1 and out.stride(1) == 1 and out.dtype == proj.dtype
    assert ba.dtype == torch.float32 and ring.dtype == torch.float32 and state.dtype == torch.float32
    assert state.is_contiguous() and ring.is_contiguous() and state.shape == (B, H, dv, dk)
    assert ring.shape == (B, m.conv, 2 * G * dk + H * dv)
    step = T == 1
    a = _DeltaParams()
    a.B, a.T, a.H, a.G, a.dk, a.dv, a.taps = B, T, H, G, dk, dv, m.conv
    a.proj, a.ldp = _p(proj), proj.stride(0)
    a.off_q, a.off_k, a.off_v, a.off_g = offs
    a.ba, a.ldba, a.off_a = _p(ba), ba.stride(0), off_a
    a.conv_q, a.conv_k, a.conv_v = _p(w["conv_q"]), _p(w["conv_k"]), _p(w["conv_v"])
    a.a_log, a.dt_bias, a.norm_w = _p(w["a_log"]), _p(w["dt_bias"]), _p(w["norm"])
    a.ring, a.state = _p(ring), _p(state)
    if not step:
        f32 = dict(device=dev, dtype=torch.float32)
        q, k = torch.empty(rows, G, dk, **f32), torch.empty(rows, G, dk, **f32)
        v, o = torch.empty(rows, H, dv, **f32), torch.empty(rows, H, dv, **f32)
        gb = torch.empty(rows, H, 2, **f32)
        a.q, a.k, a.v, a.gb, a.o = _p(q), _p(k), _p(v), _p(gb), _p(o)
    a.out, a.ldo, a.eps, a.q_scale, a.pos = _p(out), out.stride(0), eps, dk ** -0.5, _p(pos)
    _lib.call("ra_delta_mixer", ctypes.byref(a), int(step), int(proj.dtype == torch.float32), _lib.stream_ptr(),
              n_kernels=1 if step else 3)


class _LatentParams(ctypes.Structure):
    _fields_ = [("B", c_i), ("T", c_i), ("H", c_i), ("dn", c_i), ("dr", c_i), ("dv", c_i), ("r", c_i),
                ("r_pad", c_i), ("row_w", c_i), ("rot_dims", c_i),
                ("proj", c_vp), ("ldp", c_ll), ("off_q", c_i), ("off_c", c_i), ("off_g", c_i),
                ("c_norm", c_vp), ("inv_freq", c_vp), ("cache", c_vp), ("S_max", c_ll),
                ("w_uk", c_vp), ("w_uv", c_vp), ("ldw", c_ll), ("sink", c_vp),
                ("q_lat", c_vp), ("o_part", c_vp), ("lse_part", c_vp), ("splits", c_i),
                ("out", c_vp), ("ldo", c_ll), ("eps", c_f), ("scale", c_f), ("pos", c_vp)]


def latent_splits(rows: int, heads: int, n_rows: int) -> int:
    """Row ranges of the split-KV pass: enough CTAs for the machine, at least 64 cached rows each."""
    return max(1, min((n_rows + 63) // 64, 32, (148 * 8) // max(1, rows * heads)))


def latent_mixer(proj, out, *, B: int, T: int, m, offs, w, cache, n_rows: int, eps: float, pos) -> None:
    """Latent attention of ``T`` new tokens of each of ``B`` sequences over the cached rows, which the new tokens join.

    ``proj (B*T, ld)``: query heads, [latent | shared key] and output gates at columns ``offs`` (the rotated query parts are
    turned in place). ``cache (B, S_max, row)``; ``n_rows``: an upper bound of the rows that will be visible (sizes the
    grid only). ``w``: ``c_norm``, ``inv_freq``, ``uk``, ``uv``, ``sink``. ``m``: a
    :class:`~ringattention_b200.config.LatentAttentionConfig`."""
    dev = proj.device
    rows, H = B * T, m.heads
    assert proj.shape[0] == rows and proj.stride(1) == 1 and out.stride(1) == 1 and out.dtype == proj.dtype
    assert cache.is_contiguous() and cache.dtype == proj.dtype and cache.shape[0] == B
    assert w["uk"].stride(0) == w["uv"].stride(0)
    a = _LatentParams()
    a.B, a.T, a.H, a.dn, a.dr, a.dv, a.r = B, T, H, m.dim, m.rot_dim, m.vdim, m.kv_rank
    a.r_pad, a.row_w, a.rot_dims = (m.kv_rank + 7) // 8 * 8, cache.shape[2], m.rot.dims
    a.proj, a.ldp = _p(proj), proj.stride(0)
    a.off_q, a.off_c, a.off_g = offs
    a.c_norm, a.inv_freq, a.cache, a.S_max = _p(w["c_norm"]), _p(w["inv_freq"]), _p(cache), cache.shape[1]
    a.w_uk, a.w_uv, a.ldw, a.sink = _p(w["uk"]), _p(w["uv"]), w["uk"].stride(0), _p(w["sink"])
    a.splits = latent_splits(rows, H, n_rows)
    f32 = dict(device=dev, dtype=torch.float32)
    q_lat = torch.empty(rows, H, a.row_w, **f32)
    o_part = torch.empty(rows, H, a.splits, m.kv_rank, **f32)
    lse = torch.empty(rows, H, a.splits, **f32)
    a.q_lat, a.o_part, a.lse_part = _p(q_lat), _p(o_part), _p(lse)
    a.out, a.ldo, a.eps, a.scale, a.pos = _p(out), out.stride(0), eps, m.scale, _p(pos)
    is32 = int(proj.dtype == torch.float32)
    _lib.call("ra_latent_prep", ctypes.byref(a), is32, _lib.stream_ptr())
    _lib.call("ra_latent_absorbed", ctypes.byref(a), is32, _lib.stream_ptr(), n_kernels=3)
