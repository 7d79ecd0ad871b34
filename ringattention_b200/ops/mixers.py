"""Bindings of the token mixers of hybrid decoders: the gated delta rule (``delta_sm100.cu``), latent attention
(``latent_sm100.cu``) and windowed attention (``window_sm100.cu``). Activations and weights are bf16 or fp32 throughout (one type per call); states, decays, scores
and softmax are fp32 in both."""
from __future__ import annotations

import ctypes
import os

import torch

from . import _lib
from . import kernels as K

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
                ("out", c_vp), ("ldo", c_ll), ("eps", c_f), ("q_scale", c_f), ("pos", c_vp),
                ("n_chunks", c_i), ("ws_qk", c_vp), ("ws_w", c_vp), ("ws_u", c_vp), ("ws_m", c_vp), ("ws_d", c_vp),
                ("status", c_vp)]


# From this many tokens per step on the recurrence runs in chunks on the tensor cores (bf16 engines; 32-bit operands as
# sums of two bf16 numbers); below, and in fp32 engines, token by token on the CUDA cores.
CHUNK_MIN_TOKENS = int(os.environ.get("RINGATTN_B200_DELTA_CHUNK_MIN_TOKENS", "48"))
CHUNK = 64


def delta_chunk_fits(m, proj, offs) -> bool:
    """Sizes the chunked kernels take."""
    return (proj.dtype == torch.bfloat16 and m.dim in (64, 128) and m.vdim in (64, 128) and m.conv <= 4
            and not any(o % 4 for o in offs) and proj.stride(0) % 4 == 0 and proj.data_ptr() % 16 == 0)


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
    a.out, a.ldo, a.eps, a.q_scale, a.pos = _p(out), out.stride(0), eps, dk ** -0.5, _p(pos)
    entries = ("ra_delta_step",)
    if not step:
        f32 = dict(device=dev, dtype=torch.float32)
        o = torch.empty(rows, H, dv, **f32)
        a.o = _p(o)
        if T >= CHUNK_MIN_TOKENS and delta_chunk_fits(m, proj, offs):
            n = a.n_chunks = (T + CHUNK - 1) // CHUNK
            u8 = dict(device=dev, dtype=torch.uint8)
            ws = (torch.empty(B, G, n, 8 * CHUNK * dk, **u8), torch.empty(B, H, n, 4 * CHUNK * dk, **u8),
                  torch.empty(B, H, n, dv * CHUNK, **f32), torch.empty(B, H, n, 4 * CHUNK * CHUNK + 4 * CHUNK, **u8),
                  torch.empty(B, H, n, CHUNK + 4, **f32))
            a.ws_qk, a.ws_w, a.ws_u, a.ws_m, a.ws_d = (_p(t) for t in ws)
            a.status = _lib.status_tensor(dev).data_ptr()
            entries = ("ra_delta_chunk_prep", "ra_delta_chunk_scan", "ra_delta_out")
        else:
            q, k = torch.empty(rows, G, dk, **f32), torch.empty(rows, G, dk, **f32)
            v, gb = torch.empty(rows, H, dv, **f32), torch.empty(rows, H, 2, **f32)
            a.q, a.k, a.v, a.gb = _p(q), _p(k), _p(v), _p(gb)
            entries = ("ra_delta_prep", "ra_delta_scan", "ra_delta_out")
    for entry in entries:
        _lib.call(entry, ctypes.byref(a), int(proj.dtype == torch.float32), _lib.stream_ptr())


class _LatentParams(ctypes.Structure):
    _fields_ = [("B", c_i), ("T", c_i), ("H", c_i), ("dn", c_i), ("dr", c_i), ("dv", c_i), ("r", c_i),
                ("r_pad", c_i), ("row_w", c_i), ("rot_dims", c_i),
                ("proj", c_vp), ("ldp", c_ll), ("off_q", c_i), ("off_c", c_i), ("off_g", c_i),
                ("c_norm", c_vp), ("inv_freq", c_vp), ("cache", c_vp), ("S_max", c_ll),
                ("w_uk", c_vp), ("w_uv", c_vp), ("ldw", c_ll), ("sink", c_vp),
                ("q_lat", c_vp), ("o_part", c_vp), ("lse_part", c_vp), ("splits", c_i),
                ("out", c_vp), ("ldo", c_ll), ("eps", c_f), ("scale", c_f), ("pos", c_vp), ("status", c_vp)]


def latent_few_fits(m, proj, cache, w) -> bool:
    """Sizes the tensor-core kernels for few tokens take."""
    return (proj.dtype == torch.bfloat16 and m.kv_rank % 16 == 0 and m.kv_rank <= 512 and cache.shape[2] % 16 == 0
            and cache.shape[2] <= 576 and m.rot_dim % 2 == 0 and 1 <= m.dim <= 1024 and w["uk"].stride(0) % 8 == 0
            and w["uk"].data_ptr() % 16 == 0 and w["uv"].data_ptr() % 16 == 0)


def _latent_few(a, m, rows: int, B: int, T: int, n_rows: int, dev) -> None:
    """A step of few tokens on the tensor cores: 16 or 32 (token, head) rows per CTA over a range of the cache."""
    H = m.heads
    blocks = (T * H + 15) // 16 if T * H <= 16 else (T * H + 31) // 32
    tiles = (n_rows + 63) // 64
    a.splits = max(1, min((tiles + 1) // 2, 148 // (blocks * B)))
    q_lat = torch.empty(rows, H, a.row_w, device=dev, dtype=torch.bfloat16)
    o_part = torch.empty(rows, H, a.splits, m.kv_rank, device=dev, dtype=torch.float32)
    lse = torch.empty(rows, H, a.splits, device=dev, dtype=torch.float32)
    a.q_lat, a.o_part, a.lse_part, a.status = _p(q_lat), _p(o_part), _p(lse), _lib.status_tensor(dev).data_ptr()
    for entry in ("ra_latent_few_query", "ra_latent_few_attend", "ra_latent_few_output"):
        _lib.call(entry, ctypes.byref(a), _lib.stream_ptr())


def latent_splits(rows: int, heads: int, n_rows: int) -> int:
    """Row ranges of the split-KV pass: enough CTAs for the machine, at least 64 cached rows each."""
    return max(1, min((n_rows + 63) // 64, 32, (148 * 8) // max(1, rows * heads)))


def latent_mixer(proj, out, *, B: int, T: int, m, offs, w, cache, n_rows: int, eps: float, pos) -> None:
    """Latent attention of ``T`` new tokens of each of ``B`` sequences over the cached rows, which the new tokens join.

    ``proj (B*T, ld)``: query heads, [latent | shared key] and output gates at columns ``offs`` (the rotated query parts are
    turned in place). ``cache (B, S_max, row)``; ``n_rows``: the rows that will be visible, or for a single token an upper
    bound of them (it sizes grids; the kernels take the count from ``pos``). ``w``: ``c_norm``, ``inv_freq``, ``ukv`` with
    its parts ``uk`` and ``uv``, ``sink``. ``m``: a :class:`~ringattention_b200.config.LatentAttentionConfig`."""
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
    a.out, a.ldo, a.eps, a.scale, a.pos = _p(out), out.stride(0), eps, m.scale, _p(pos)
    a.splits, is32 = 1, int(proj.dtype == torch.float32)
    expand = T >= EXPAND_MIN_TOKENS and two_part_fits(m, proj, out, offs)
    if not expand and latent_few_fits(m, proj, cache, w):
        return _latent_few(a, m, rows, B, T, n_rows, proj.device)
    _lib.call("ra_latent_prep", ctypes.byref(a), is32, _lib.stream_ptr())
    if expand:
        return _latent_expanded(proj, out, B, T, m, offs, w, cache, n_rows)
    f32 = dict(device=proj.device, dtype=torch.float32)
    a.splits = latent_splits(rows, H, n_rows)
    q_lat = torch.empty(rows, H, a.row_w, **f32)
    o_part = torch.empty(rows, H, a.splits, m.kv_rank, **f32)
    lse = torch.empty(rows, H, a.splits, **f32)
    a.q_lat, a.o_part, a.lse_part = _p(q_lat), _p(o_part), _p(lse)
    _lib.call("ra_latent_absorbed", ctypes.byref(a), is32, _lib.stream_ptr(), n_kernels=3)


# From this many tokens of a sequence per step on, keys and values are made from the cached latents (one product over all
# of them, H (dim + vdim) columns) and the tensor-core attention runs per head; below, the queries go to the latents.
EXPAND_MIN_TOKENS = int(os.environ.get("RINGATTN_B200_LATENT_EXPAND_MIN_TOKENS", "96"))


class _TwoPartArgs(ctypes.Structure):
    _fields_ = [("q", c_vp), ("q_sb", c_ll), ("q_ss", c_ll), ("q_sh", c_ll),
                ("k1", c_vp), ("k1_sb", c_ll), ("k1_ss", c_ll), ("k1_sh", c_ll),
                ("k2", c_vp), ("k2_sb", c_ll), ("k2_ss", c_ll),
                ("v", c_vp), ("v_sb", c_ll), ("v_ss", c_ll), ("v_sh", c_ll),
                ("out", c_vp), ("o_sb", c_ll), ("o_ss", c_ll), ("o_sh", c_ll),
                ("sink", c_vp), ("gate", c_vp), ("gate_ld", c_ll),
                ("B", c_i), ("H", c_i), ("Sq", c_i), ("Sk", c_i), ("d1", c_i), ("d2", c_i), ("dv", c_i),
                ("scale", c_f), ("q_pos0", c_i), ("status", c_vp), ("stream", c_vp)]


def two_part_attention(q, k1, k2, v, out, *, scale: float, q_pos0: int, sink=None, gate=None) -> None:
    """Causal attention on the tensor cores with two-part keys: ``score = (q1 . k1 + q2 . k2) * scale``.

    ``q (B, Sq, H, d1 + d2)``, ``k1 (B, Sk, H, d1)``, ``k2 (B, Sk, d2)`` shared by the heads, ``v (B, Sk, H, dv)``, ``out (B, Sq,
    H, dv)``: bf16 views, innermost contiguous. Query i sits at position ``q_pos0 + i``. ``sink (H,)`` fp32: one more entry
    ``exp(sink)`` in each denominator; ``gate (B*Sq, H)``: bf16 view, the head's output is multiplied by its sigmoid."""
    B, Sq, H, _ = q.shape
    a = _TwoPartArgs()
    a.q, (a.q_sb, a.q_ss, a.q_sh) = _p(q), q.stride()[:3]
    a.k1, (a.k1_sb, a.k1_ss, a.k1_sh) = _p(k1), k1.stride()[:3]
    a.k2, (a.k2_sb, a.k2_ss) = _p(k2), k2.stride()[:2]
    a.v, (a.v_sb, a.v_ss, a.v_sh) = _p(v), v.stride()[:3]
    a.out, (a.o_sb, a.o_ss, a.o_sh) = _p(out), out.stride()[:3]
    a.sink, a.gate, a.gate_ld = _p(sink), _p(gate), 0 if gate is None else gate.stride(0)
    a.B, a.H, a.Sq, a.Sk = B, H, Sq, k1.shape[1]
    a.d1, a.d2, a.dv = k1.shape[3], k2.shape[2], v.shape[3]
    a.scale, a.q_pos0 = scale, q_pos0
    a.status, a.stream = _lib.status_tensor(q.device).data_ptr(), torch.cuda.current_stream().cuda_stream
    _lib.call("ra_attn_two_part", ctypes.byref(a))


def two_part_fits(m, proj, out, offs) -> bool:
    """Sizes the tensor-core kernel takes (every part starts at a multiple of 16 bytes)."""
    return (proj.dtype == torch.bfloat16 and 8 <= m.dim <= 128 and 8 <= m.rot_dim <= 64 and 8 <= m.vdim <= 128
            and not (m.dim % 8 or m.rot_dim % 8 or m.vdim % 8 or offs[0] % 8 or proj.stride(0) % 8 or out.stride(0) % 8
                     or out.data_ptr() % 16))


def _latent_expanded(proj, out, B: int, T: int, m, offs, w, cache, n: int) -> None:
    H, dn, dr, dv = m.heads, m.dim, m.rot_dim, m.vdim
    S_max, width = cache.shape[1:]
    r_pad = (m.kv_rank + 7) // 8 * 8
    kv = torch.empty(B, n, w["ukv"].shape[0], device=proj.device, dtype=proj.dtype)
    for b in range(B):
        K.linear_ex(cache[b, :n, :r_pad], w["ukv"], kv[b])
    ld = proj.stride(0)
    q = proj.as_strided((B, T, H, dn + dr), (T * ld, ld, dn + dr, 1), proj.storage_offset() + offs[0])
    o = out.as_strided((B, T, H, dv), (T * out.stride(0), out.stride(0), dv, 1), out.storage_offset())
    two_part_attention(q, kv[:, :, :H * dn].view(B, n, H, dn), cache[:, :n, r_pad:r_pad + dr],
                       kv[:, :, w["uv_off"]:w["uv_off"] + H * dv].view(B, n, H, dv), o, scale=m.scale, q_pos0=n - T,
                       sink=w["sink"], gate=proj[:, offs[2]:offs[2] + H])


# --------------------------------------------------------------------------------------------- windowed attention
class _WindowParams(ctypes.Structure):
    _fields_ = [("B", c_i), ("T", c_i), ("H", c_i), ("G", c_i), ("dk", c_i), ("dv", c_i), ("rot_half", c_i),
                ("proj", c_vp), ("ldp", c_ll), ("off_q", c_i), ("off_k", c_i), ("off_v", c_i),
                ("q_norm", c_vp), ("k_norm", c_vp), ("inv_freq", c_vp), ("k_cache", c_vp), ("v_cache", c_vp),
                ("R", c_i), ("kw", c_i), ("vw", c_i), ("window", c_i), ("sink", c_vp), ("out", c_vp), ("ldo", c_ll),
                ("eps", c_f), ("scale", c_f), ("pos", c_vp), ("splits", c_i), ("n_max", c_ll)]


class _WindowArgs(ctypes.Structure):
    _fields_ = [("q", c_vp), ("q_sb", c_ll), ("q_ss", c_ll), ("q_sh", c_ll),
                ("k", c_vp), ("k_sb", c_ll), ("k_ss", c_ll), ("k_sh", c_ll),
                ("v", c_vp), ("v_sb", c_ll), ("v_ss", c_ll), ("v_sh", c_ll),
                ("out", c_vp), ("o_sb", c_ll), ("o_ss", c_ll), ("o_sh", c_ll), ("sink", c_vp),
                ("B", c_i), ("H", c_i), ("G", c_i), ("Sq", c_i), ("dk", c_i), ("dv", c_i), ("window", c_i), ("k_rows", c_i),
                ("scale", c_f), ("q_pos0", c_ll), ("status", c_vp), ("stream", c_vp)]


def window_attention(q, k_ring, v_ring, out, *, scale: float, q_pos0: int, window: int, sink) -> None:
    """Causal attention over the last ``window`` keys on the tensor cores. ``q (B, Sq, H, dk)`` at positions ``q_pos0 ..``,
    ``k_ring (B, G, R, dk)`` and ``v_ring (B, G, R, dv)`` with position p in row ``p % R``, ``out (B, Sq, H, dv)``: bf16 views,
    innermost contiguous; ``sink (H,)`` fp32. The ring has to hold the window of every query of the step."""
    B, Sq, H, dk = q.shape
    a = _WindowArgs()
    a.q, (a.q_sb, a.q_ss, a.q_sh) = _p(q), q.stride()[:3]
    a.k, (a.k_sb, a.k_sh, a.k_ss) = _p(k_ring), k_ring.stride()[:3]
    a.v, (a.v_sb, a.v_sh, a.v_ss) = _p(v_ring), v_ring.stride()[:3]
    a.out, (a.o_sb, a.o_ss, a.o_sh) = _p(out), out.stride()[:3]
    a.sink, a.B, a.H, a.G, a.Sq, a.dk, a.dv = _p(sink), B, H, k_ring.shape[1], Sq, dk, v_ring.shape[3]
    a.window, a.k_rows, a.scale, a.q_pos0 = window, k_ring.shape[2], scale, q_pos0
    a.status, a.stream = _lib.status_tensor(q.device).data_ptr(), torch.cuda.current_stream().cuda_stream
    _lib.call("ra_attn_window", ctypes.byref(a))


def window_tensor_core_fits(m, proj, out) -> bool:
    """Sizes the tensor-core kernels take (every head starts at a multiple of 16 bytes)."""
    return (proj.dtype == torch.bfloat16 and m.dim <= 128 and m.vdim <= 128 and not (m.dim % 8 or m.vdim % 8)
            and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0)


def window_mixer(proj, out, *, B: int, T: int, m, offs, w, cache, length: int, eps: float, pos) -> None:
    """Windowed attention of ``T`` new tokens of each of ``B`` sequences.

    ``proj (B*T, ld)``: query, key and value projections at columns ``offs`` (queries are normed and turned in place).
    ``cache``: a :class:`~ringattention_b200.models.cache.WindowCache`, which the new tokens join. ``length``: tokens before
    this step (for a single token an upper bound that sizes grids; the kernels take positions from ``pos``). ``w``: ``q_norm``,
    ``k_norm``, ``inv_freq``, ``sink``. ``m``: a :class:`~ringattention_b200.config.WindowAttentionConfig`."""
    rows, H, G, dk, dv = B * T, m.heads, m.kv_heads, m.dim, m.vdim
    assert proj.shape[0] == rows and proj.stride(1) == 1 and out.stride(1) == 1 and out.dtype == proj.dtype
    assert cache.k.is_contiguous() and cache.v.is_contiguous() and cache.k.dtype == proj.dtype
    a = _WindowParams()
    a.B, a.T, a.H, a.G, a.dk, a.dv, a.rot_half = B, T, H, G, dk, dv, m.rot.dims // 2
    a.proj, a.ldp = _p(proj), proj.stride(0)
    a.off_q, a.off_k, a.off_v = offs
    a.q_norm, a.k_norm, a.inv_freq, a.sink = _p(w["q_norm"]), _p(w["k_norm"]), _p(w["inv_freq"]), _p(w["sink"])
    a.k_cache, a.v_cache, a.R, a.kw, a.vw = _p(cache.k), _p(cache.v), cache.rows, cache.k.shape[3], cache.v.shape[3]
    a.window = min(cache.window, 1 << 30)
    a.out, a.ldo, a.eps, a.scale, a.pos, a.n_max = _p(out), out.stride(0), eps, m.scale, _p(pos), length + 1
    is32, fits = int(proj.dtype == torch.float32), window_tensor_core_fits(m, proj, out)
    if T == 1 and fits:
        return _lib.call("ra_window_decode", ctypes.byref(a), _lib.stream_ptr())
    _lib.call("ra_window_prep", ctypes.byref(a), is32, _lib.stream_ptr())
    if not fits:
        return _lib.call("ra_window_attend", ctypes.byref(a), is32, _lib.stream_ptr())
    ld = proj.stride(0)
    q = proj.as_strided((B, T, H, dk), (T * ld, ld, dk, 1), proj.storage_offset() + offs[0])
    o = out.as_strided((B, T, H, dv), (T * out.stride(0), out.stride(0), dv, 1), out.storage_offset())
    window_attention(q, cache.k, cache.v, o, scale=m.scale, q_pos0=length, window=a.window, sink=w["sink"])
