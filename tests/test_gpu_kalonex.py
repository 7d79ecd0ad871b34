"""Kalonex decoders (windowed attention with a sink, routed experts, looped layers) on the GPU against the plain
implementation: mechanisms alone, whole prompts, decoding, portions, windows and rings, reuse of caches, batches, long
decoding, and generation through the engine."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import kalonex_torch as R
from kalonex_configs import CONFIGS, layer, model, moe

pytestmark = pytest.mark.gpu

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# rms of the logits' error over the rms of the logits
TOL = {torch.float32: 2e-5, torch.bfloat16: 0.06}
BOTH = [torch.float32, torch.bfloat16]


def engine(raw, w, dtype, ctx=1024, batch=1, max_step=8192):
    from ringattention_b200.config import HybridConfig
    from ringattention_b200.models import registry

    return registry.make_engine(HybridConfig.from_dict(raw), ctx, source=w, dtype=dtype, batch=batch, max_step=max_step)


def row_errors(got, want):
    """Per row: rms of the centred difference over the rms of the centred reference."""
    from ringattention_b200.ops import _lib

    _lib.check_status()
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    d = got - want
    d, c = d - d.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / c.pow(2).mean().sqrt()


def check_logits(name, dtype, got, want):
    """bf16 may swap two experts with nearly equal scores, which changes that token: there some rows may be off."""
    e = row_errors(got, want)
    if name == "routed" and dtype == torch.bfloat16:
        assert e.quantile(0.75) < TOL[dtype] and e.median() < TOL[dtype] / 2
    else:
        assert e.max() < TOL[dtype]


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


def feed(eng, tok, sizes):
    """Run ``tok`` through ``eng`` in steps of the given sizes (the last size repeats); single tokens decode."""
    out, i, n = [], 0, 0
    while i < len(tok):
        s = min(sizes[min(n, len(sizes) - 1)], len(tok) - i)
        part = tok[None, i:i + s].cuda()
        out.append(eng.decode_step(part[:, 0]) if s == 1 and i > 0 else eng.step(part)[0])
        i, n = i + s, n + 1
    return torch.cat(out)


# ---------------------------------------------------------------------------------------------- products and rows
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("M", [1, 3, 8, 9, 200])
def test_bias_scale_and_gated_products(dtype, M):
    from ringattention_b200.ops import kernels as K

    torch.manual_seed(M)
    Kd, N, F = 136, 88, 72
    x = torch.randn(M, Kd, device="cuda").to(dtype)
    w = (torch.randn(N, Kd, device="cuda") / Kd ** 0.5).to(dtype)
    b = torch.zeros(96, device="cuda")
    b[:N] = torch.randn(N, device="cuda") * 3
    ref = x.double() @ w.double().t()
    tol = 1e-5 if dtype == torch.float32 else 3e-2
    out = K.linear_ex(x, w, torch.empty(M, N, device="cuda", dtype=dtype), bias=b)
    assert (out.double() - ref - b[:N].double()).abs().max() < tol * 3
    res = torch.randn(M, N, device="cuda")
    acc = res.clone()
    K.linear_ex(x, w, acc, residual=acc, bias=b)
    assert (acc.double() - ref - b[:N].double() - res.double()).abs().max() < 1e-4
    zero = torch.zeros(96, device="cuda")
    out = K.linear_ex(x, w, torch.empty(M, N, device="cuda"), bias=zero, alpha=0.37)
    assert (out.double() - 0.37 * ref).abs().max() < 1e-4
    with pytest.raises(AssertionError):
        K.linear_ex(x, w, torch.empty(M, N, device="cuda"), alpha=2.0)
    gu = (torch.randn(2 * F, Kd, device="cuda") / Kd ** 0.5).to(dtype)
    wide = torch.full((M, F + 16), 7.0, device="cuda", dtype=dtype)
    K.linear_gated(x, gu, wide[:, 8:8 + F])
    g, u = (x.double() @ gu.double().t()).split(F, dim=1)
    want = R.silu(g) * u
    assert ((wide[:, 8:8 + F].double() - want).abs() < tol * (1 + want.abs())).all()
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + F:] == 7).all()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("d", [36, 107, 512])
def test_stream_beside_embedding(dtype, d):
    from ringattention_b200.models.weights import round8
    from ringattention_b200.ops import kernels as K

    dp = round8(d)
    table = torch.randn(50, d, device="cuda").to(dtype)
    x = torch.zeros(7, dp, device="cuda")
    x[:, :d] = torch.randn(7, d, device="cuda")
    tok = torch.tensor([0, 49, 3, 3, 20, 1, 48], device="cuda", dtype=torch.int32)
    out = K.stream_pair(tok, table, x, d)
    assert torch.equal(out[:, :dp], x.to(dtype)) and torch.equal(out[:, dp:dp + d], table[tok.long()])
    assert (out[:, dp + d:] == 0).all()


# ---------------------------------------------------------------------------------------------- attention alone
# heads, kv_heads, dim, vdim, window, rotary dims
SHAPES = [(6, 2, 20, 28, 5, 6), (4, 2, 128, 64, 130, 64), (3, 3, 64, 128, 128, 0), (16, 1, 64, 64, 200, 32),
          (40, 2, 48, 40, 33, 16), (8, 8, 128, 128, 1, 128), (2, 1, 160, 136, 90, 80), (5, 1, 8, 24, 129, 8),
          (32, 8, 128, 128, 70, 64), (48, 2, 128, 64, 90, 0), (72, 8, 112, 16, 50, 48)]


def attention_setup(shape, dtype, T, seed=0):
    from ringattention_b200.config import HybridConfig

    H, G, D, Dv, win, rot = shape
    raw = model(8, 8, [layer(H, G, D, Dv, win, rot, 1.3 * D ** -0.5, None)], (0, 1, 1))
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype)
    q, k, v = rnd(T, H * D), rnd(T, G * D), rnd(T, G * Dv)
    qn, kn = (1 + 0.3 * rnd(H * D).float()).to(dtype), (1 + 0.3 * rnd(G * D).float()).to(dtype)
    sink = torch.randn(H, generator=g)
    return HybridConfig.from_dict(raw).layers[0].mixer, [q, k, v, qn, kn, sink]


def attention_reference(m, t, eps=1e-5, window=None):
    q, k, v, qn, kn, sink = [x.double() for x in t]
    T, pos = q.shape[0], torch.arange(q.shape[0])
    turn = lambda x, w, h: R.rotate_half(R.norm(x, w, eps).view(T, h, -1), pos, m.rot.base, m.rot.dims)
    return R.attention_core(turn(q, qn, m.heads), turn(k, kn, m.kv_heads), v.view(T, m.kv_heads, m.vdim), m.scale,
                            m.window if window is None else window, sink).reshape(T, -1)


def run_attention(m, t, dtype, sizes, max_step, context, eps=1e-5):
    """The mixer over the sequence in portions, through a ring for steps of at most ``max_step`` tokens."""
    from ringattention_b200.models.cache import WindowCache
    from ringattention_b200.models.weights import round8
    from ringattention_b200.ops import mixers as X

    q, k, v, qn, kn, sink = t
    H, D, Dv, G = m.heads, m.dim, m.vdim, m.kv_heads
    offs = (0, round8(H * D), round8(H * D) + round8(G * D))
    proj = torch.zeros(q.shape[0], offs[2] + round8(G * Dv), device="cuda", dtype=dtype)
    for o, x in zip(offs, (q, k, v)):
        proj[:, o:o + x.shape[1]] = x.cuda()
    w = {"q_norm": qn.cuda(), "k_norm": kn.cuda(), "sink": sink.cuda(),
         "inv_freq": torch.tensor(m.rot.inv_freq(), dtype=torch.float64).float().cuda()}
    cache = WindowCache(m, 1, context, max_step, "cuda", dtype)
    out = torch.zeros(q.shape[0], round8(H * Dv), device="cuda", dtype=dtype)
    i, n = 0, 0
    while i < q.shape[0]:
        s = min(sizes[min(n, len(sizes) - 1)], q.shape[0] - i)
        assert s <= max_step
        X.window_mixer(proj[i:i + s], out[i:i + s, :H * Dv], B=1, T=s, m=m, offs=offs, w=w, cache=cache, length=i, eps=eps,
                       pos=torch.tensor([i, 0], device="cuda", dtype=torch.int64))
        i, n = i + s, n + 1
    return out[:, :H * Dv], cache


def attention_error(m, t, dtype, sizes, max_step=8192, context=1024):
    from ringattention_b200.ops import _lib

    got, _ = run_attention(m, t, dtype, sizes, max_step, context)
    _lib.check_status()
    assert torch.isfinite(got).all()
    return (got.double().cpu() - attention_reference(m, t)).abs().max().item()


ATT_TOL = {torch.float32: 5e-5, torch.bfloat16: 3e-2}  # (32-bit angles are off by some 1e-5 at these positions)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_alone(dtype, shape):
    m, t = attention_setup(shape, dtype, 420)
    for sizes in ([420], [1], [2], [3, 129, 1, 64], [128, 127, 2, 1], [300, 1]):
        assert attention_error(m, t, dtype, sizes) < ATT_TOL[dtype]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", SHAPES[:6])
def test_ring_goes_round_several_times(dtype, shape):
    """A ring of a few tiles: rows are used again and again, in portions and token by token."""
    m, t = attention_setup(shape, dtype, 1000, seed=1)
    for sizes in ([40], [64, 1, 17, 2], [50, 1]):
        got, cache = run_attention(m, t, dtype, sizes, 64, 4096)
        assert cache.rows <= 512
        # (32-bit angles are off by about 1e-4 at positions around a thousand)
        assert (got.double().cpu() - attention_reference(m, t)).abs().max() < max(ATT_TOL[dtype], 2e-4)


def stand_out(m, t, i, j):
    """Key j and query i of every head point the same way in a dimension that does not turn: with the returned mixer the
    score of the pair is 20, far above all others."""
    q, k, v, qn, kn, _ = t
    D = m.dim
    qn[:], kn[:] = 1, 1
    q[i] *= 0.05
    k[j] *= 0.05
    q.view(q.shape[0], m.heads, D)[i, :, D - 1] = 9
    k.view(k.shape[0], m.kv_heads, D)[j, :, D - 1] = 9
    v[j] = 4
    return m.__class__(**{**m.__dict__, "scale": 20 / D})


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(4, 2, 128, 64, 130, 64), (6, 2, 20, 28, 70, 6), (16, 1, 64, 64, 128, 32)])
def test_windows_edge(dtype, shape):
    """A pair that stands out, just inside and just outside the window, in a prompt, at a portion's start and decoded."""
    win, i = shape[4], 391
    for back in (0, 1, win - 2, win - 1, win, win + 1, i):
        m, t = attention_setup(shape, dtype, 400, seed=2)
        m = stand_out(m, t, i, i - back)
        ref = attention_reference(m, t)
        assert ((ref[i] - 4).abs().max() < 0.2) == (back < win)
        if back in (win - 1, win):  # the pair shows: a window that is one off changes the row
            other = attention_reference(m, t, window=win - 1 if back < win else win + 1)
            assert (ref - other)[i].abs().max() > 1
        for sizes in ([400], [i, 9], [i, 1], [i - 1, 2, 1], [i - win + 1, 1], [100, 1]):
            got, _ = run_attention(m, t, dtype, sizes, 400, 1024)
            assert (got.double().cpu() - ref).abs().max() < 2 * ATT_TOL[dtype]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(4, 2, 128, 64, 130, 64), (6, 2, 20, 28, 7, 6), (40, 2, 48, 40, 33, 16)])
def test_sink_and_first_tokens(dtype, shape):
    """Sinks from nothing to everything; the sink is not scaled and counts once, also for the first token."""
    for value in (-40.0, -1.0, 0.0, 3.0, 30.0):
        m, t = attention_setup(shape, dtype, 140, seed=4)
        t[5] = t[5] * 0.5 + value
        for sizes in ([140], [1], [2, 1], [5, 3, 1]):
            assert attention_error(m, t, dtype, sizes) < ATT_TOL[dtype]
    big = attention_reference(m, t)
    assert big[0].abs().max() < 1e-3                   # nothing is left beside the largest sink
    t[5] = t[5] * 0 - 60
    assert torch.allclose(attention_reference(m, t)[0].view(m.heads, -1)[0], t[2][0].double().view(m.kv_heads, -1)[0])


# ---------------------------------------------------------------------------------------------- experts alone
def experts_setup(E, top, ff, shared, d, rows, dtype, seed=0, one_expert=None):
    from ringattention_b200.config import HybridConfig
    from ringattention_b200.models.weights import HybridWeights

    raw = model(8, d, [layer(1, 1, 8, 8, 4, 2, 1.0, moe(E, top, ff, shared))], (0, 1, 1))
    w = R.random_model(raw, seed=seed)
    if one_expert is not None:      # a constant input dimension makes every token choose it first
        w["l0.mlp.router"][:, 0] = -3
        w["l0.mlp.router"][one_expert, 0] = 4
    cfg = HybridConfig.from_dict(raw)
    W = HybridWeights(cfg, w.__getitem__, dtype, "cuda")
    h = torch.zeros(rows, W.dp, dtype=dtype)
    h[:, :d] = torch.randn(rows, d, generator=torch.Generator().manual_seed(seed + 1)).to(dtype)
    if one_expert is not None:
        h[:, 0] = 4
    ref = R.experts(h[:, :d].double(), {n: t.to(dtype).double() for n, t in w.items()}, "l0.mlp.", raw["layers"][0]["mlp"])
    return cfg.layers[0].mlp, W, h.cuda(), ref


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("E, top, ff, shared, d", [(5, 2, 36, 20, 108), (37, 4, 72, None, 64), (1, 1, 8, 8, 40),
                                                   (64, 8, 136, 264, 192), (3, 3, 300, 40, 72), (130, 1, 16, None, 136)])
def test_experts_alone(dtype, E, top, ff, shared, d):
    from ringattention_b200.ops import _lib, experts

    for rows in (1, 4, 8, 9, 64, 333):
        m, W, h, ref = experts_setup(E, top, ff, shared, d, rows, dtype, seed=rows)
        x0 = torch.zeros(rows, W.dp, device="cuda")
        x0[:, :d] = torch.randn(rows, d, device="cuda")
        x = x0.clone()
        experts.moe_(x, h, d, m, W.layers[0].moe)
        _lib.check_status()
        err = ((x - x0)[:, :d].double().cpu() - ref).abs().max(-1).values
        assert err.max() < (1e-4 if dtype == torch.float32 else 0.06) * max(1.0, ref.abs().max().item() / 3)
        assert (x[:, d:] == 0).all()


@pytest.mark.parametrize("dtype", BOTH)
def test_all_tokens_choose_one_expert(dtype):
    """Lists of unequal length: one expert has every token, some have none."""
    from ringattention_b200.ops import _lib, experts

    m, W, h, ref = experts_setup(20, 1, 48, 16, 96, 300, dtype, one_expert=13)
    x = torch.zeros(300, W.dp, device="cuda")
    experts.moe_(x, h, 96, m, W.layers[0].moe)
    _lib.check_status()
    assert (x[:, :96].double().cpu() - ref).abs().max() < (1e-3 if dtype == torch.float32 else 0.05 * ref.abs().max())


def test_score_multiplies_the_input():
    """With a score well below one the places differ: silu(w g) (w u) is not w silu(g) u."""
    m, W, h, ref = experts_setup(4, 2, 24, None, 48, 16, torch.float32)
    raw = model(8, 48, [layer(1, 1, 8, 8, 4, 2, 1.0, moe(4, 2, 24))], (0, 1, 1))
    raw_w = {n: t.double() for n, t in R.random_model(raw, seed=0).items()}
    hd = h.cpu().double()[:, :48]
    chosen, weight = R.route(hd, raw_w["l0.mlp.router"], 2)
    after = torch.zeros_like(hd)
    for t in range(16):
        for e, s in zip(chosen[t].tolist(), weight[t]):
            after[t] += s * R.gated(hd[t], raw_w, f"l0.mlp.e{e}.")
    assert (after - ref).abs().max() > 0.1


# ---------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("sizes", [[10000], [1], [2], [3, 130, 1, 64], [128, 127, 2, 1], [259, 1]])
def test_prompt_in_any_portions(dtype, name, sizes):
    raw, w, tok, ref = oracle(name, 260)
    check_logits(name, dtype, feed(engine(raw, w, dtype), tok, sizes), ref)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["odd", "fused"])
def test_layer_run_by_layer_run(dtype, name):
    """Every run of a looped layer has its own cache, and the pass's vector and product come right before its first layer."""
    raw, w, tok, _ = oracle(name, 260)
    want, got = [], []
    R.forward(raw, w, tok.tolist(), want)
    engine(raw, w, dtype).step(tok[None].cuda(), taps=got)
    loop = raw["loop"]
    assert len(got) == len(want) == len(raw["layers"]) + (loop["times"] - 1) * (loop["stop"] - loop["start"])
    for a, b in zip(got, want):
        assert (a.double().cpu() - b).abs().max() < (1e-4 if dtype == torch.float32 else 0.08) * b.abs().max()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["odd", "fused", "ones"])
def test_rings_smaller_than_the_prompt(dtype, name):
    """Steps longer than a ring takes are cut; the logits asked for come in the order asked for."""
    raw, w, tok, ref = oracle(name, 260)
    eng = engine(raw, w, dtype, max_step=48)
    assert min(c.rows for c in eng.caches) < 260
    assert row_errors(eng.step(tok[None].cuda())[0], ref).max() < TOL[dtype]
    eng.reset()
    eng.step(tok[None, :100].cuda(), want=[])
    got = eng.step(tok[None, 100:].cuda(), want=[159, 0, 47, 48, 48])[0]
    assert row_errors(got, ref[[259, 100, 147, 148, 148]]).max() < TOL[dtype]
    eng.reset()
    assert row_errors(feed(eng, tok, [30, 1]), ref).max() < TOL[dtype]


@pytest.mark.parametrize("dtype", BOTH)
def test_caches_are_used_again(dtype):
    raw, w, tok, ref = oracle("fused", 260)
    eng = engine(raw, w, dtype, ctx=300)
    noise = torch.randint(0, raw["vocab"], (1, 300), generator=torch.Generator().manual_seed(9))
    for length in (300, 1, 129):
        eng.step(noise[:, :length].cuda(), want=[])
        eng.reset()
        assert row_errors(feed(eng, tok, [100, 3, 1]), ref).max() < TOL[dtype]
        eng.reset()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["odd", "fused"])
@pytest.mark.parametrize("batch", [3, 11])
def test_batch_of_sequences_against_each_alone(dtype, name, batch):
    raw, w, tok, ref = oracle(name, 260)
    n = 90
    rows = torch.stack([tok[13 * b:13 * b + n] for b in range(batch)])
    eng = engine(raw, w, dtype, batch=batch, ctx=200)
    out = [eng.step(rows[:, :60].cuda()), eng.step(rows[:, 60:62].cuda())]
    out += [eng.decode_step(rows[:, i].cuda())[:, None] for i in range(62, n)]
    got = torch.cat(out, dim=1)
    for b in (0, 1, batch - 1):
        assert row_errors(got[b], R.forward(raw, w, rows[b].tolist())).max() < TOL[dtype]


@pytest.mark.parametrize("name", ["odd", "fused"])
def test_long_decoding_through_the_graph(name):
    """Greedy tokens of ``generate`` (graph replay) are the plain implementation's up to near-ties."""
    raw, w, tok, _ = oracle(name, 260)
    for dtype in BOTH:
        eng = engine(raw, w, dtype, ctx=512, max_step=64)
        gen, _ = eng.generate(tok[None, :37].cuda(), 300, chunk=20)
        seq = tok[:37].tolist() + gen[0].tolist()
        ref = R.forward(raw, w, seq[:-1])[36:]
        best, mine = ref.max(-1).values, ref.gather(1, gen[0].cpu()[:, None])[:, 0]
        slack = (2e-4 if dtype == torch.float32 else 0.5) * ref.std()
        assert gen.shape == (1, 300) and (best - mine < slack).all()


def test_command_line_generates_and_replays(tmp_path):
    """The program that replays token ids gives the engine's logits; the generation program runs on the same folder."""
    from ringattention_b200.models.weights import write_safetensors

    raw, w, tok, ref = oracle("fused", 260)
    (tmp_path / "config.json").write_text(json.dumps(raw))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tok[:200].tolist(), "want": [199, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tok[200:202].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tok[202:203].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": tok[:1].tolist(), "want": [0]}], "end": ["b"]}]
    for name, dtype in (("float32", torch.float32), ("bfloat16", torch.bfloat16)):
        r = subprocess.run([os.path.join(REPO, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", name, "--out",
                            str(tmp_path), "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps),
                           capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(
            -1, raw["vocab"])
        got = torch.cat([read(0), read(2), read(3)])
        assert row_errors(got, ref[[199, 3, 202, 0]]).max() < TOL[dtype] and not (tmp_path / "1.f32").exists()
    r = subprocess.run([sys.executable, os.path.join(REPO, "infer.py"), "--model", str(tmp_path), "--context", "150", "--chunk",
                        "64", "--new-tokens", "6"], capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    out = json.loads(r.stdout.splitlines()[-1])
    assert out["decode_tokens_per_s"] > 0 and math.isfinite(out["prefill_tokens_per_s"])
