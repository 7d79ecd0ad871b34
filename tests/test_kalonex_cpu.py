"""Host side of the Kalonex decoders: configuration, registry, packing, the rings' sizes, order of the layer runs, and the
plain implementation's own mechanisms against even plainer statements of them."""
import json
import math

import pytest
import torch

import kalonex_torch as R
from kalonex_configs import CONFIGS, FUSED, ODD, ROUTED


def parse(raw):
    from ringattention_b200.config import HybridConfig

    return HybridConfig.from_dict(raw)


def test_config_from_dict():
    from ringattention_b200.config import DenseConfig, MoEConfig, WindowAttentionConfig

    c = parse(ODD)
    assert all(isinstance(l.mixer, WindowAttentionConfig) for l in c.layers)
    assert c.layers[0].mlp == DenseConfig(90, gated=True) and c.layers[1].mlp == MoEConfig(5, 5, 36, 20)
    assert c.layers[2].mlp is None and parse(ROUTED).layers[0].mlp.shared_ff == 64
    m = c.layers[1].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.scale, m.rot.dims) == (3, 3, 12, 20, 33, 0.4, 12)
    assert c.logit_scale == 0.3 and c.norm_gain_offset == 0 and not c.design.parallel and c.rms_eps == 1e-4
    raw = json.loads(json.dumps(ODD))
    raw["layers"][0]["mixer"]["mask"] = None
    assert parse(raw).layers[0].mixer.window is None


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_order_of_the_layer_runs(name):
    raw = CONFIGS[name]
    assert [(r.layer, r.enter) for r in parse(raw).runs] == R.schedule(raw)


def test_order_by_hand():
    c = parse(FUSED)
    assert [(r.layer, r.enter) for r in c.runs] == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None)]
    assert [(r.layer, r.enter) for r in parse(ROUTED).runs] == [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]


@pytest.mark.parametrize("change, match", [
    (lambda c: c["layers"][0].update(type="delta"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotary"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "window"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "experts"),
    (lambda c: c["loop"].update(stop=4), "loop"),
    (lambda c: c["loop"].update(start=2), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
])
def test_config_rejects(change, match):
    c = json.loads(json.dumps(ODD))
    change(c)
    with pytest.raises(ValueError, match=match):
        parse(c)


def test_registry_and_presets(tmp_path):
    from ringattention_b200.config import LlamaConfig
    from ringattention_b200.models import registry

    (tmp_path / "config.json").write_text(json.dumps(FUSED))
    c = registry.load_config(str(tmp_path))
    assert c == parse(FUSED) and registry.family_of(c) is registry.FAMILIES["Kalonex"]
    assert {torch.bfloat16, torch.float32} == set(registry.family_of(c).dtypes)
    for name, partner in (("kalonex-1b", "llama-1b"), ("kalonex-7b", "llama-7b")):
        c, l = registry.load_config(name, n_layers=8), LlamaConfig.named(partner, n_layers=8)
        assert len(c.runs) == 8 and c.d_model == l.d_model and c.architecture == "Kalonex"
        f = c.layers[1].mlp                            # as wide per token as the dense layers
        assert f.top * f.ff + f.shared_ff == c.layers[0].mlp.ff == l.d_ff
    with pytest.raises(ValueError, match="layer runs"):
        registry.load_config("kalonex-1b", n_layers=5)


def test_number_of_parameters():
    for raw in CONFIGS.values():
        n = sum(math.prod(s) for name, s in R.shapes(raw).items() if len(s) == 2 and name != "loop.step")
        assert parse(raw).n_params() == n


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_packed_weights_hold_every_tensor(name):
    """The packed matrices contain each tensor at its place and zeros everywhere else."""
    from ringattention_b200.models.weights import HybridWeights, hybrid_tensor_shapes, round8

    raw = CONFIGS[name]
    cfg, w = parse(raw), R.random_model(raw, seed=1)
    assert hybrid_tensor_shapes(cfg) == {n: tuple(t.shape) for n, t in w.items()}
    W = HybridWeights(cfg, w.__getitem__, torch.float32, "cpu")
    d, dp = cfg.d_model, W.dp

    def holds(packed, parts):
        seen = torch.zeros_like(packed)
        for r, c, t in parts:
            seen[r:r + t.shape[0], c:c + t.shape[1]] = t
        return torch.equal(seen, packed)

    def gated(gu, down, p):
        g, u, dn = (w[p + n].float() for n in ("gate", "up", "down"))
        return holds(gu, [(0, 0, g), (round8(g.shape[0]), 0, u)]) and holds(down, [(0, 0, dn)])

    for i, L in W.layers.items():
        p = f"l{i}.mix."
        assert all(o % 8 == 0 for o in L.offs)
        assert holds(L.in_w, [(o, 0, w[p + n].float()) for o, n in zip(L.offs, "qkv")])
        assert holds(L.in_b[:, None], [(o, 0, w[p + n + ".b"].float()[:, None]) for o, n in zip(L.offs, "qkv")])
        assert L.in_b.numel() % 32 == 0 and L.in_b.numel() >= L.in_w.shape[0]
        assert holds(L.out_w, [(0, 0, w[p + "o"].float())]) and holds(L.out_b[:, None], [(0, 0, w[p + "o.b"].float()[:, None])])
        f, p = cfg.layers[i].mlp, f"l{i}.mlp."
        if f is None:
            assert L.moe is None and L.gu_w is None
        elif L.moe is None:
            assert gated(L.gu_w, L.down_w, p)
        else:
            assert all(gated(L.moe["gu"][e], L.moe["down"][e], f"{p}e{e}.") for e in range(f.experts))
            assert holds(L.moe["router"], [(0, 0, w[p + "router"].float())])
            assert ("sh_gu" in L.moe) == (f.shared_ff is not None)
            assert f.shared_ff is None or gated(L.moe["sh_gu"], L.moe["sh_down"], p + "shared.")
    lin = w["loop.in"].float()
    assert holds(W.loop_w, [(0, 0, lin[:, :d]), (0, dp, lin[:, d:])])
    assert all(torch.equal(s[:d], t) and (s[d:] == 0).all() for s, t in zip(W.loop_step, w["loop.step"].float()))
    with pytest.raises(ValueError, match="shape"):
        HybridWeights(cfg, lambda n: w[n][:1], torch.float32, "cpu")


def test_rings_hold_a_steps_windows():
    """Whatever the position, the keys of a step from a tile border on fit in the ring without meeting."""
    from ringattention_b200.models.cache import WindowCache

    m = parse(FUSED).layers[0].mixer                   # window 130
    for context, max_step in ((100, 8192), (5000, 1), (5000, 64), (5000, 127), (5000, 1000), (1024, 8192)):
        c = WindowCache(m, 1, context, max_step, "cpu", torch.float32)
        assert c.rows % 128 == 0 and c.rows <= (context + 127) // 128 * 128
        for pos in range(0, context, 37):
            T = min(max_step, context - pos)
            first = max(0, pos - m.window + 1) // 128 * 128
            assert pos + T - first <= c.rows
    assert WindowCache(m, 1, 100000, 64, "cpu", torch.float32).rows == 384
    cfg = parse(FUSED)
    assert cfg.cache_bytes(1 << 20, max_step=64) < cfg.cache_bytes(1 << 20) == cfg.cache_bytes(1 << 20, max_step=1 << 20)


def test_long_steps_are_cut_and_put_together():
    """Places asked for across the portions of a step come back in the order asked for."""
    from ringattention_b200.models.hybrid_infer import HybridInference

    class Fake(HybridInference):
        def __init__(self):
            self.B, self.max_step, self.calls = 1, 10, []

        def step(self, tokens, want=None, taps=None):
            self.calls.append(tokens.shape[1])
            return tokens[:, want, None].float() if len(want) else None

    eng, tok = Fake(), torch.arange(35)[None]
    assert eng._long_step(tok, [34, 0, 9, 10, 0], None)[0, :, 0].tolist() == [34, 0, 9, 10, 0]
    assert eng.calls == [10, 10, 10, 5]
    assert eng._long_step(tok, None, None)[0, :, 0].tolist() == list(range(35)) and eng._long_step(tok, [], None) is None
    with pytest.raises(ValueError, match="taps"):
        eng._long_step(tok, None, [])


# ---------------------------------------------------------------------------------------------- the plain implementation
def test_oracle_rotation_by_hand():
    x = torch.zeros(1, 1, 6, dtype=torch.float64)
    x[0, 0, 0], x[0, 0, 4], x[0, 0, 5] = 1.0, 2.0, 3.0
    y = R.rotate_half(x, torch.tensor([1]), 500.0, 4)
    assert torch.allclose(y[0, 0], torch.tensor([math.cos(1), 0, math.sin(1), 0, 2, 3], dtype=torch.float64))
    a, b = torch.randn(1, 1, 8, dtype=torch.float64), torch.randn(1, 1, 8, dtype=torch.float64)
    rot = lambda v, p: R.rotate_half(v, torch.tensor([p]), 500.0, 8)
    assert torch.allclose((rot(a, 3) * rot(b, 10)).sum(), (rot(a, 40) * rot(b, 47)).sum())


def test_oracle_window_and_sink_by_hand():
    assert R.window_mask(4, 2).tolist() == [[True, False, False, False], [True, True, False, False],
                                            [False, True, True, False], [False, False, True, True]]
    s = torch.tensor([[[1.0, 9.0], [2.0, 3.0]]], dtype=torch.float64)
    p = R.sink_softmax(s, R.window_mask(2, 2), torch.tensor([0.5], dtype=torch.float64))
    e = [math.exp(x) for x in (1, 2, 3, 0.5)]
    want = [[e[0] / (e[0] + e[3]), 0], [e[1] / (e[1] + e[2] + e[3]), e[2] / (e[1] + e[2] + e[3])]]
    assert torch.allclose(p[0], torch.tensor(want, dtype=torch.float64))


def test_oracle_groups_of_heads():
    torch.manual_seed(0)
    q, k, v = (torch.randn(5, h, 3, dtype=torch.float64) for h in (4, 2, 2))
    sink = torch.randn(4, dtype=torch.float64)
    whole = R.attention_core(q, k, v, 0.7, 3, sink)
    for h in range(4):
        one = R.attention_core(q[:, h:h + 1], k[:, h // 2:h // 2 + 1], v[:, h // 2:h // 2 + 1], 0.7, 3, sink[h:h + 1])
        assert torch.allclose(whole[:, h:h + 1], one)


def test_oracle_routing_by_hand():
    w = torch.eye(4, dtype=torch.float64)
    chosen, weight = R.route(torch.tensor([[0.1, -2.0, 3.0, 0.5]], dtype=torch.float64), w, 2)
    assert chosen.tolist() == [[2, 3]]
    assert torch.allclose(weight, torch.tensor([[1 / (1 + math.exp(-3)), 1 / (1 + math.exp(-0.5))]], dtype=torch.float64))


def test_oracle_pass_enters_with_stream_first():
    w = {"loop.in": torch.tensor([[1.0, 0, 10, 0], [0, 1, 0, 10]]), "loop.step": torch.tensor([[0.0, 0], [0.5, -0.5]])}
    y = R.enter_pass(torch.tensor([[1.0, 2.0]]), torch.tensor([[3.0, 4.0]]), w, 1)
    assert y.tolist() == [[31.5, 41.5]]


def test_oracle_planted_mistakes_show():
    """A window that is one token off, a sink left out, biases left out and a pass too few change the logits of a model of
    the kind the other tests use."""
    w = R.random_model(ODD, seed=0)
    tok = torch.randint(0, ODD["vocab"], (60,), generator=torch.Generator().manual_seed(0)).tolist()
    ref = R.forward(ODD, w, tok)
    far = lambda raw, weights: (R.forward(raw, weights, tok) - ref).pow(2).mean().sqrt() / ref.std()
    off = json.loads(json.dumps(ODD))
    off["layers"][0]["mixer"]["mask"]["size"] += 1
    once = json.loads(json.dumps(ODD))
    once["loop"]["times"] = 1
    without = lambda end: {n: t * 0 if n.endswith(end) else t for n, t in w.items()}
    for raw, weights in ((off, w), (once, w), (ODD, {**w, **{n: t * 0 - 60 for n, t in w.items() if n.endswith("sink")}}),
                         (ODD, without("k.b")), (ODD, without("v.b")), (ODD, without("o.b")), (ODD, without("loop.step"))):
        assert far(raw, weights) > 0.02
