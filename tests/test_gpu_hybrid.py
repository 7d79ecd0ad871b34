"""Hybrid decoders (gated delta rule, latent attention) on the GPU against the plain implementation: mechanisms alone,
whole prompts, decoding, portions, reuse of cache and states, long decoding, and generation through the engine."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import dafelorn_torch as R
from hybrid_configs import CONFIGS, ONES, TWO_KINDS, WIDE, latent, model

pytestmark = pytest.mark.gpu

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# rms of the logits' error over the rms of the logits
TOL = {torch.float32: 2e-5, torch.bfloat16: 0.06}
BOTH = [torch.float32, torch.bfloat16]


def engine(raw, w, dtype, ctx=1024, batch=1):
    from ringattention_b200.config import HybridConfig
    from ringattention_b200.models import registry

    return registry.make_engine(HybridConfig.from_dict(raw), ctx, source=w, dtype=dtype, batch=batch)


def error(got, want):
    """Worst row: rms of the centred difference over the rms of the centred reference."""
    from ringattention_b200.ops import _lib

    _lib.check_status()
    got, want = got.double().cpu(), want.double()
    assert torch.isfinite(got).all()
    d = got - want
    d, c = d - d.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / c.pow(2).mean().sqrt()).max().item()


_MODELS = {}


def oracle(name, T, seed=3):
    """(raw config, weights, tokens, logits) of a named configuration; computed once."""
    key = (name, T, seed)
    if key not in _MODELS:
        raw = CONFIGS[name]
        w = R.random_model(raw, seed=seed)
        tok = torch.randint(0, raw["vocab"], (T,), generator=torch.Generator().manual_seed(seed))
        _MODELS[key] = raw, w, tok, R.forward(raw, w, tok.tolist())
    return _MODELS[key]


def feed(eng, tok, sizes, end=None):
    """Run ``tok`` through ``eng`` in steps of the given sizes (the last size repeats); single tokens decode."""
    out, i, n = [], 0, 0
    while i < len(tok):
        s = min(sizes[min(n, len(sizes) - 1)], len(tok) - i)
        part = tok[None, i:i + s].cuda()
        out.append(eng.decode_step(part[:, 0]) if s == 1 and i > 0 else eng.step(part)[0])
        i, n = i + s, n + 1
    return torch.cat(out)


# ---------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("d", [36, 108, 4096, 5000])
def test_two_norms_of_one_stream(dtype, d):
    from ringattention_b200.models.weights import round8
    from ringattention_b200.ops import kernels as K

    torch.manual_seed(0)
    dp = round8(d)
    x = torch.zeros(9, dp, device="cuda")
    x[:, :d] = torch.randn(9, d, device="cuda") * torch.tensor([1e-3, 1, 50] * 3, device="cuda")[:, None]
    w = [torch.zeros(dp, device="cuda", dtype=dtype) for _ in range(2)]
    for t in w:
        t[:d] = torch.randn(d, device="cuda") * 0.3
    idx = torch.tensor([8, 1, 1, 0], dtype=torch.int32, device="cuda")
    for rows in (None, idx):
        y = K.norm_f32(x, d, 1e-4, 1.0, w[0], w[1], rows_idx=rows)
        src = x.double().cpu() if rows is None else x.double().cpu()[rows.long().cpu()]
        for got, g in zip(y, w):
            ref = R.zero_centred_norm(src[:, :d], g.double().cpu()[:d], 1e-4)
            assert (got[:, :d].double().cpu() - ref).abs().max() <= (1e-5 if dtype == torch.float32 else 0.01) * ref.abs().max()
            assert (got[:, d:] == 0).all()
    y1, y2 = K.norm_f32(x, d, 1e-4, 0.0, w[0])         # plain gain, one output
    assert y2 is None
    ref = R.rms(x.double().cpu()[:, :d], 1e-4) * w[0].double().cpu()[:d]
    assert (y1[:, :d].double().cpu() - ref).abs().max() <= (1e-5 if dtype == torch.float32 else 0.01) * ref.abs().max()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("M", [1, 2, 5, 8, 9, 200])
def test_linear_epilogues(dtype, M):
    """Addend in fp32, squared relu, and a tail of columns in fp32, for a handful of rows and for many."""
    from ringattention_b200.ops import kernels as K

    torch.manual_seed(M)
    tol = 1e-5 if dtype == torch.float32 else 0.01
    for N, Kd in ((72, 40), (328, 520)):
        x = torch.randn(M, Kd, device="cuda").to(dtype)
        w = (torch.randn(N, Kd, device="cuda") / math.sqrt(Kd)).to(dtype)
        ref = x.double() @ w.double().t()
        wide = torch.full((M, N + 16), float("nan"), device="cuda", dtype=dtype)
        K.linear_ex(x, w, wide[:, 8:8 + N], relu2=True)
        assert (wide[:, 8:8 + N].double() - R.relu_squared(ref)).abs().max() <= tol * R.relu_squared(ref).abs().max()
        assert wide[:, :8].isnan().all() and wide[:, 8 + N:].isnan().all()
        r = torch.randn(M, N, device="cuda")
        want = ref + r.double()
        K.linear_ex(x, w, r, residual=r)
        assert (r.double() - want).abs().max() <= tol / 10 * want.abs().max() + 1e-5
        main, tail = torch.empty(M, 64, device="cuda", dtype=dtype), torch.empty(M, N - 64, device="cuda")
        K.linear_ex(x, w, main, tail=tail, n_split=64)
        assert (main.double() - ref[:, :64]).abs().max() <= tol * ref.abs().max()
        assert (tail.double() - ref[:, 64:]).abs().max() <= 1e-4 * ref.abs().max()
    _status()


def _status():
    from ringattention_b200.ops import _lib

    _lib.check_status()


def run_delta(m, proj, ba, w, state, ring, pos, sizes, dtype, eps):
    """Feed ``proj (T, q|k|v|g)`` through the mixer in steps; offsets as given by the sizes (padded to 8)."""
    from ringattention_b200.ops import mixers as X

    outs, i, n = [], 0, 0
    r8 = lambda v: (v + 7) // 8 * 8
    G, dk, H, dv = m.kv_heads, m.dim, m.heads, m.vdim
    offs = (0, r8(G * dk), 2 * r8(G * dk), 2 * r8(G * dk) + r8(H * dv))
    while i < proj.shape[0]:
        s = min(sizes[min(n, len(sizes) - 1)], proj.shape[0] - i)
        out = torch.empty(s, H * dv, device="cuda", dtype=dtype)
        p = torch.tensor([pos + i, 0], dtype=torch.int64, device="cuda")
        X.delta_mixer(proj[i:i + s].contiguous(), ba[i:i + s].contiguous(), out, B=1, T=s, m=m, offs=offs, off_a=r8(H),
                      w=w, ring=ring, state=state, eps=eps, pos=p)
        outs.append(out)
        i, n = i + s, n + 1
    _status()
    return torch.cat(outs), offs


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(6, 2, 24, 40, 4), (4, 4, 128, 128, 3), (2, 1, 200, 24, 2), (3, 3, 64, 96, 1), (4, 2, 128, 64, 4), (5, 1, 64, 128, 2),
                                   (2, 2, 64, 64, 1), (40, 20, 128, 128, 4)])
def test_delta_mixer_alone(dtype, shape):
    """Decays from almost 0 to almost 1, large and small step sizes, repeated keys (where the delta rule differs most from
    a plain sum), whole and in pieces, with the state carried on."""
    from ringattention_b200.config import GatedDeltaConfig

    H, G, dk, dv, taps = shape
    m = GatedDeltaConfig(H, G, dk, dv, taps)
    T = 150
    g = torch.Generator().manual_seed(sum(shape))
    rn = lambda *s: torch.randn(*s, generator=g)
    r8 = lambda v: (v + 7) // 8 * 8
    wid = 2 * r8(G * dk) + 2 * r8(H * dv)
    proj = rn(T, wid)
    proj[70:90] = proj[70:71]                          # the same key again and again
    proj = proj.to(dtype)
    ba = torch.zeros(T, 2 * r8(H))
    ba[:, :H], ba[:, r8(H):r8(H) + H] = 2 * rn(T, H), 2 * rn(T, H)
    w = {"conv_q": rn(G * dk, taps), "conv_k": rn(G * dk, taps), "conv_v": rn(H * dv, taps),
         "a_log": torch.linspace(-5, 2, H), "dt_bias": rn(H), "norm": 1 + 0.2 * rn(dv)}
    w = {n: t.to(dtype) for n, t in w.items()}
    # reference
    f = {n: t.double() for n, t in w.items()}
    P = proj.double()
    oq, ok, ov, og = 0, r8(G * dk), 2 * r8(G * dk), 2 * r8(G * dk) + r8(H * dv)
    q, k, v = (R.silu(R.causal_conv(P[:, o:o + n], f[c])) for o, n, c in
               ((oq, G * dk, "conv_q"), (ok, G * dk, "conv_k"), (ov, H * dv, "conv_v")))
    q = (R.unit(q.view(T, G, dk)) * dk ** -0.5).repeat_interleave(H // G, 1)
    k = R.unit(k.view(T, G, dk)).repeat_interleave(H // G, 1)
    beta = torch.sigmoid(ba[:, :H].double())
    gam = torch.exp(-torch.exp(f["a_log"]) * R.softplus(ba[:, r8(H):r8(H) + H].double() + f["dt_bias"]))
    o, S = R.gated_delta_scan(q, k, v.view(T, H, dv), gam, beta)
    want = (R.rms(o, 1e-5) * f["norm"] * R.silu(P[:, og:og + H * dv].view(T, H, dv))).reshape(T, H * dv)
    wc = {n: t.cuda() for n, t in w.items()}
    for sizes in ([T], [64, 63, 1], [2, 3, 5, 17], [1], [100, 2]):
        state = torch.zeros(1, H, dv, dk, device="cuda")
        ring = torch.full((1, taps, 2 * G * dk + H * dv), float("nan"), device="cuda")   # rows of no token are never read
        got, _ = run_delta(m, proj.cuda(), ba.cuda(), wc, state, ring, 0, sizes, dtype, 1e-5)
        tol = 2e-4 if dtype == torch.float32 else 0.02
        assert (got.double().cpu() - want).abs().max() <= tol * want.abs().max(), sizes
        # the state is fp32 in both types: the order of its sums, and in the chunked form the two-term operands, differ
        assert (state[0].double().cpu() - S.transpose(1, 2)).abs().max() <= 2e-4 * S.abs().max(), sizes


def latent_case(H, dn, dr, dv, r, T, dtype, seed, scale=0.2, base=100.0):
    from ringattention_b200.config import LatentAttentionConfig, RotaryConfig

    m = LatentAttentionConfig(H, dn, dr, dv, r, scale, RotaryConfig(base, dr))
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g)
    r8 = lambda v: (v + 7) // 8 * 8
    offs = (0, r8(H * (dn + dr)), r8(H * (dn + dr)) + r8(r + dr))
    proj = rn(T, offs[2] + r8(H)).to(dtype)
    lw = r8(r)
    uk, uv = torch.zeros(H * dn, lw), torch.zeros(H * dv, lw)
    uk[:, :r], uv[:, :r] = rn(H * dn, r) / math.sqrt(r), rn(H * dv, r) / math.sqrt(r)
    w = {"c_norm": (1 + 0.2 * rn(r)).to(dtype), "inv_freq": torch.tensor(m.rot.inv_freq(), dtype=torch.float32),
         "sink": torch.linspace(-1, 2, H)}
    both = torch.zeros(r8(H * dn) + r8(H * dv), lw)
    both[:H * dn], both[r8(H * dn):r8(H * dn) + H * dv] = uk, uv
    w["ukv"], w["uv_off"] = both.to(dtype), r8(H * dn)
    return m, offs, proj, w


def latent_want(m, offs, proj, w, eps):
    H, dn, dr, dv, r = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
    T = proj.shape[0]
    P = proj.double()
    pos = torch.arange(T)
    c = R.rms(P[:, offs[1]:offs[1] + r], eps) * w["c_norm"].double()
    q = P[:, :H * (dn + dr)].view(T, H, dn + dr)
    kr = R.rotate_interleaved(P[:, offs[1] + r:offs[1] + r + dr], pos, m.rot.base, dr)
    qr = R.rotate_interleaved(q[..., dn:], pos, m.rot.base, dr)
    kv = w["ukv"].double()
    k = (c @ kv[:H * dn, :r].t()).view(T, H, dn)
    v = (c @ kv[w["uv_off"]:w["uv_off"] + H * dv, :r].t()).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :dn], k) + torch.einsum("ihd,jd->hij", qr, kr)) * m.scale
    p = R.sink_softmax(s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf), w["sink"].double())
    o = torch.einsum("hij,jhd->ihd", p, v)
    return (o * torch.sigmoid(P[:, offs[2]:offs[2] + H])[..., None]).reshape(T, H * dv), p


def run_latent(m, offs, proj, w, sizes, dtype, eps, ctx):
    from ringattention_b200.config import LatentAttentionConfig  # noqa: F401
    from ringattention_b200.models.cache import LatentCache
    from ringattention_b200.ops import mixers as X

    cache = LatentCache(m, 1, ctx, "cuda", dtype)
    cache.data.fill_(float("nan"))                     # rows of no token are never used
    wc = {n: t.cuda() if torch.is_tensor(t) else t for n, t in w.items()}
    wc["uk"], wc["uv"] = wc["ukv"][:m.heads * m.dim], wc["ukv"][w["uv_off"]:w["uv_off"] + m.heads * m.vdim]
    outs, i, n = [], 0, 0
    while i < proj.shape[0]:
        s = min(sizes[min(n, len(sizes) - 1)], proj.shape[0] - i)
        out = torch.empty(s, m.heads * m.vdim, device="cuda", dtype=dtype)
        p = torch.tensor([i, 0], dtype=torch.int64, device="cuda")
        X.latent_mixer(proj[i:i + s].cuda().contiguous(), out, B=1, T=s, m=m, offs=offs, w=wc, cache=cache.data,
                       n_rows=i + s if s > 1 else ctx, eps=eps, pos=p)
        outs.append(out)
        i, n = i + s, n + 1
    _status()
    return torch.cat(outs)


LATENT_SHAPES = [(3, 20, 6, 28, 52), (4, 128, 64, 128, 256), (16, 128, 64, 128, 512), (5, 64, 32, 64, 128), (1, 16, 2, 8, 24),
                 (2, 48, 16, 96, 80), (20, 40, 24, 32, 208), (33, 24, 8, 16, 40), (16, 32, 16, 24, 16)]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_latent_mixer_alone(dtype, shape):
    T = 333
    m, offs, proj, w = latent_case(*shape, T, dtype, seed=sum(shape))
    want, _ = latent_want(m, offs, proj, w, 1e-5)
    for sizes in ([T], [200, 100, 31, 1], [64, 2, 3, 7, 128], [300, 1]):
        got = run_latent(m, offs, proj, w, sizes, dtype, 1e-5, ctx=T)   # the last token fills the cache to the brim
        tol = 5e-5 if dtype == torch.float32 else 0.02
        assert (got.double().cpu() - want).abs().max() <= tol * want.abs().max(), sizes


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(3, 20, 6, 28, 52), (4, 128, 64, 128, 256)])
@pytest.mark.parametrize("key", [0, 1, 63, 64, 127, 128, 255, 256, 299])
def test_one_far_key_stands_out(dtype, shape, key):
    """One latent is made so that the late queries give it much of their weight: a key left out or taken twice at the
    border of a tile or split would change the whole output."""
    H, dn, dr, dv, r = shape
    T = 420
    m, offs, proj, w = latent_case(*shape, T, dtype, seed=5)
    uk = w["ukv"][:H * dn, :r].double()
    c = R.rms(proj[:, offs[1]:offs[1] + r].double(), 1e-5) * w["c_norm"].double()
    k = (c[key] @ uk.t()).view(H, dn)
    late = slice(400, T)
    aim = k / k.norm(dim=-1, keepdim=True) * (16.0 / m.scale / k.norm(dim=-1, keepdim=True))
    q = proj[late, :H * (dn + dr)].view(-1, H, dn + dr)
    q[..., :dn] = aim.to(dtype)
    q[..., dn:] *= 0.1
    want, p = latent_want(m, offs, proj, w, 1e-5)
    assert p[:, late, key].mean() > 0.2
    for sizes in ([T], [400, 20], [400, 1], [410, 5, 1]):
        got = run_latent(m, offs, proj, w, sizes, dtype, 1e-5, ctx=512)
        tol = 5e-5 if dtype == torch.float32 else 0.02
        assert (got.double().cpu() - want).abs().max() <= tol * want.abs().max(), sizes


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(3, 20, 6, 28, 52), (4, 128, 64, 128, 256)])
def test_sink_and_first_tokens(dtype, shape):
    """Scores near zero and sinks from negligible to dominant; the first tokens see one, two, ... keys."""
    m, offs, proj, w = latent_case(*shape, 140, dtype, seed=9, scale=0.01)
    w["sink"] = torch.linspace(-20.0, 6.0, shape[0])
    want, _ = latent_want(m, offs, proj, w, 1e-5)
    for sizes in ([140], [1], [2, 1, 1, 2]):
        got = run_latent(m, offs, proj, w, sizes, dtype, 1e-5, ctx=256)
        err = (got.double().cpu() - want).abs().view(140, shape[0], -1).amax(-1)
        ref = want.abs().view(140, shape[0], -1).amax(-1)
        assert (err <= (5e-5 if dtype == torch.float32 else 0.03) * ref + 1e-7).all()


# ---------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("sizes", [[10000], [1], [2], [3, 130, 1, 64], [128, 127, 2, 1], [299, 1]])
def test_prompt_in_any_portions(dtype, name, sizes):
    raw, w, tok, want = oracle(name, 310)
    got = feed(engine(raw, w, dtype, ctx=310), tok, sizes)
    assert error(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", BOTH)
def test_layer_by_layer(dtype):
    raw, w, tok, _ = oracle("two_kinds", 310)
    ref, taps = [], []
    R.forward(raw, w, tok[:40].tolist(), taps=ref)
    engine(raw, w, dtype).step(tok[None, :40].cuda(), taps=taps)
    assert len(ref) == len(taps) == len(raw["layers"])
    for a, b in zip(taps, ref):
        assert (a.double().cpu() - b).abs().max() <= (2e-5 if dtype == torch.float32 else 0.03) * b.abs().max()


@pytest.mark.parametrize("dtype", BOTH)
def test_cache_and_states_are_used_again(dtype):
    """A second request after a longer first one, and after one that ended in the middle: nothing of them is left."""
    raw, w, tok, _ = oracle("two_kinds", 310)
    eng = engine(raw, w, dtype, ctx=512)
    feed(eng, tok, [250, 1])
    other = torch.flip(tok, [0])[:90]
    want = R.forward(raw, w, other.tolist())
    for sizes in ([90], [2], [40, 1]):
        eng.reset()
        assert error(feed(eng, other, sizes), want) < TOL[dtype]


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_batch_of_sequences_against_each_alone(name):
    raw, w, tok, want = oracle(name, 310)
    rows = torch.stack([tok[:100], tok[100:200], tok[200:300]])
    refs = torch.stack([R.forward(raw, w, r.tolist()) for r in rows])
    for dtype in BOTH:
        eng = engine(raw, w, dtype, ctx=128, batch=3)
        out = [eng.step(rows[:, :70].cuda()), eng.step(rows[:, 70:73].cuda())]
        out += [eng.decode_step(rows[:, i].cuda())[:, None] for i in range(73, 100)]
        got = torch.cat(out, dim=1)
        for b in range(3):
            assert error(got[b], refs[b]) < TOL[dtype]


def test_long_decoding_through_the_graph():
    """Generation through the engine's own entry point: the tokens are those of a step-by-step greedy run, and the logits of
    the whole sequence agree with the plain implementation."""
    for dtype in BOTH:
        raw, w, tok, _ = oracle("wide", 310)
        eng = engine(raw, w, dtype, ctx=512)
        gen, timing = eng.generate(tok[None, :37].cuda(), 300, chunk=16)
        assert gen.shape == (1, 300) and len(timing["decode_ms"]) == 300
        seq = torch.cat([tok[:37], gen[0].cpu()])
        want = R.forward(raw, w, seq.tolist())
        got = feed(engine(raw, w, dtype, ctx=512), seq, [37, 1])
        assert error(got, want) < TOL[dtype]
        assert torch.equal(got[36:-1].argmax(-1).cpu(), gen[0].cpu())      # every token is the greedy one
        again, _ = eng.generate(tok[None, :37].cuda(), 20, chunk=37, use_graph=False)
        if dtype == torch.float32:
            assert torch.equal(again[0], gen[0, :20])


def test_want_picks_places_and_bounds_are_checked():
    raw, w, tok, want = oracle("ones", 310)
    eng = engine(raw, w, torch.float32, ctx=64)
    got = eng.step(tok[None, :50].cuda(), want=[49, 0, 7, 7])[0]
    assert error(got, want[[49, 0, 7, 7]]) < TOL[torch.float32]
    assert eng.step(tok[None, 50:52].cuda(), want=[]) is None
    with pytest.raises(ValueError, match="max_context"):
        eng.step(tok[None, 52:80].cuda())
    with pytest.raises(ValueError, match="outside"):
        eng.step(tok[None, 52:54].cuda(), want=[2])
    assert eng.length == 52
    assert error(eng.step(tok[None, 52:64].cuda())[0], want[52:64]) < TOL[torch.float32]   # filled to the brim
    with pytest.raises(ValueError, match="max_context"):
        eng.decode_step(tok[64:65].cuda())


def test_command_line_replays_a_trace(tmp_path):
    """The replay program on a model folder, in both types, requests one after the other."""
    from ringattention_b200.models.weights import write_safetensors

    raw, w, tok, want = oracle("two_kinds", 310)
    mdl, out = tmp_path / "model", tmp_path / "out"
    mdl.mkdir()
    out.mkdir()
    (mdl / "config.json").write_text(json.dumps(raw))
    write_safetensors(str(mdl / "model.safetensors"), w)
    t = tok.tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:100], "want": [0, 99]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[100:102], "want": [1]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[102:103], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": t[:9], "want": [8]}], "end": ["y"]}]
    places = {0: [0, 99], 1: [101], 2: [102], 3: [8]}
    for dtype in ("bfloat16", "float32"):
        r = subprocess.run([sys.executable, os.path.join(REPO, "bin", "trace_run"), "--model", str(mdl), "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps),
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        for i, p in places.items():
            got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(len(p), -1)
            assert error(got, want[p]) < TOL[getattr(torch, dtype)]
