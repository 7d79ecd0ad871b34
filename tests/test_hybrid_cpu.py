"""Host side of the hybrid decoder family: configuration, registry, checkpoint reading and packing, trace protocol, and
the plain implementation's own mechanisms against even plainer statements of them."""
import io
import json
import math

import pytest
import torch

import dafelorn_torch as R
from hybrid_configs import CONFIGS, TWO_KINDS


def test_config_from_dict():
    from ringattention_b200.config import GatedDeltaConfig, HybridConfig, LatentAttentionConfig

    c = HybridConfig.from_dict(TWO_KINDS)
    assert [type(l.mixer) for l in c.layers] == [GatedDeltaConfig, LatentAttentionConfig, GatedDeltaConfig,
                                                 LatentAttentionConfig, GatedDeltaConfig]
    assert [c.owner(i) for i in range(5)] == [0, 1, 2, 1, 0]
    assert c.layers[2].mlp is None and c.layers[0].mlp.ff == 90
    assert c.rms_eps == TWO_KINDS["norm"]["eps"] and c.vocab_size == 331
    rot = c.layers[1].mixer.rot
    assert rot.inv_freq() == [rot.base ** (-2 * i / rot.dims) for i in range(rot.dims // 2)]


@pytest.mark.parametrize("change, match", [
    (lambda c: c["layers"][0].update(type="other"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "feed-forward kind"),
    (lambda c: c["layers"][3].update(weights_of=9), "not a layer"),
    (lambda c: c["layers"][3]["mixer"].update(heads=7), "other sizes"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
])
def test_config_rejects(change, match):
    from ringattention_b200.config import HybridConfig

    c = json.loads(json.dumps(TWO_KINDS))
    change(c)
    with pytest.raises(ValueError, match=match):
        HybridConfig.from_dict(c)


def test_registry(tmp_path):
    from ringattention_b200.config import HybridConfig, LlamaConfig
    from ringattention_b200.models import registry

    assert isinstance(registry.load_config("llama-tiny"), LlamaConfig)
    assert registry.load_config("dafelorn-1b", n_layers=5).n_layers == 5
    (tmp_path / "config.json").write_text(json.dumps(TWO_KINDS))
    assert isinstance(registry.load_config(str(tmp_path)), HybridConfig)
    assert torch.float32 in registry.family_of(registry.load_config(str(tmp_path))).dtypes
    assert torch.float32 not in registry.family_of(LlamaConfig()).dtypes
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Llama", "d_model": 256, "n_heads": 2}))
    assert registry.load_config(str(tmp_path)).d_model == 256
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "nobody's"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.load_config(str(tmp_path))
    with pytest.raises(KeyError):
        registry.load_config("nothing-7b")


def test_safetensors_round_trip_and_damage(tmp_path):
    from ringattention_b200.models.weights import SafetensorsFile, write_safetensors

    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 2, 2)}
    p = str(tmp_path / "m.safetensors")
    write_safetensors(p, t)
    f = SafetensorsFile(p)
    assert f.names() == list(t) and all(torch.equal(f[n], t[n]) for n in t) and "z" not in f
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-4])
    with pytest.raises(ValueError, match="does not fit"):
        SafetensorsFile(p)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_packed_weights_hold_every_tensor(name):
    """The packed matrices contain each tensor at its place and zeros everywhere else."""
    from ringattention_b200.config import HybridConfig, LatentAttentionConfig
    from ringattention_b200.models.weights import HybridWeights, hybrid_tensor_shapes

    raw = CONFIGS[name]
    cfg, w = HybridConfig.from_dict(raw), R.random_model(raw, seed=1)
    assert hybrid_tensor_shapes(cfg) == {n: tuple(t.shape) for n, t in w.items()}
    W = HybridWeights(cfg, w.__getitem__, torch.float32, "cpu")
    d = cfg.d_model
    for i, L in W.layers.items():
        m = cfg.layers[i].mixer
        names = ["q", "dkv", "g"] if isinstance(m, LatentAttentionConfig) else ["q", "k", "v", "g", "b", "a"]
        offs = list(L.offs)
        if L.n_split is not None:
            assert L.n_split % 32 == 0
            offs += [L.n_split, L.n_split + L.off_a]
        seen = torch.zeros_like(L.in_w)
        for n, o in zip(names, offs):
            t = w[f"l{i}.mix.{n}"].float()
            assert o % 8 == 0 and torch.equal(L.in_w[o:o + t.shape[0], :d], t)
            seen[o:o + t.shape[0], :d] = t
        assert torch.equal(seen, L.in_w)
        o = w[f"l{i}.mix.o"].float()
        assert torch.equal(L.out_w[:d, :o.shape[1]], o) and (L.out_w[:, o.shape[1]:L.o_cols] == 0).all()
        if cfg.layers[i].mlp is not None:
            dn = w[f"l{i}.mlp.down"].float()
            assert torch.equal(L.out_w[:d, L.o_cols:L.o_cols + dn.shape[1]], dn)
    with pytest.raises(ValueError, match="shape"):
        HybridWeights(cfg, lambda n: w[n][:1], torch.float32, "cpu")


class FakeEngine:
    """Logits of a place: [token, position, steps so far that were decode steps]."""

    device = torch.device("cpu")

    def __init__(self):
        self.length, self.resets, self.decoded = 0, 0, 0

    def reset(self):
        self.length, self.decoded = 0, 0
        self.resets += 1

    def step(self, tokens, want):
        rows = [[float(tokens[0, w]), float(self.length + w), float(self.decoded)] for w in want]
        self.length += tokens.shape[1]
        return torch.tensor([rows]) if rows else None

    def decode_step(self, tokens):
        self.decoded += 1
        self.length += 1
        return torch.tensor([[float(tokens[0]), float(self.length - 1), float(self.decoded)]])


def test_trace_runner_protocol(tmp_path):
    from ringattention_b200.utils.trace import TraceRunner

    run = TraceRunner(FakeEngine())
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [9, 10], "want": []}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": [11], "want": [0]}], "end": ["b"]}]
    for s in steps:
        run.step(s, str(tmp_path))
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).tolist()
    assert read(0) == [7, 2, 0, 5, 0, 0] and read(1) == [8, 3, 1] and not (tmp_path / "2.f32").exists()
    assert read(3) == [11, 0, 0]                       # a first token is a prompt, also when it is the only one
    run.step({"step": 4, "entries": [{"id": "c", "tokens": [1], "want": []}], "end": []}, str(tmp_path))
    for bad in ({"id": "d", "tokens": [1], "want": []}, {"id": "c", "tokens": [], "want": []},
                {"id": "c", "tokens": [1], "want": [1]}):
        with pytest.raises(ValueError):
            run.step({"step": 5, "entries": [bad], "end": []}, str(tmp_path))


def test_trace_refuses_a_type_no_engine_has(tmp_path, capsys):
    from ringattention_b200.utils import trace

    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Llama"}))
    assert trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path)]) == 3


# ---------------------------------------------------------------------------------------------- the oracle itself
def test_oracle_conv_is_causal_and_last_tap_is_now():
    x = torch.randn(6, 2, dtype=torch.float64)
    w = torch.randn(2, 3, dtype=torch.float64)
    y = R.causal_conv(x, w)
    assert torch.allclose(y[0], x[0] * w[:, 2])
    assert torch.allclose(y[4], x[4] * w[:, 2] + x[3] * w[:, 1] + x[2] * w[:, 0])


def test_oracle_scan_single_head_by_hand():
    torch.manual_seed(0)
    T, dk, dv = 5, 3, 2
    q, k, v = (torch.randn(T, 1, n, dtype=torch.float64) for n in (dk, dk, dv))
    g, b = torch.rand(T, 1, dtype=torch.float64), torch.rand(T, 1, dtype=torch.float64)
    o, S = R.gated_delta_scan(q, k, v, g, b)
    M = torch.zeros(dk, dv, dtype=torch.float64)
    for t in range(T):
        M = (torch.eye(dk, dtype=torch.float64) - b[t, 0] * torch.outer(k[t, 0], k[t, 0])) @ (g[t, 0] * M)
        M = M + b[t, 0] * torch.outer(k[t, 0], v[t, 0])
        assert torch.allclose(o[t, 0], M.t() @ q[t, 0])
    assert torch.allclose(S[0], M)


def test_oracle_sink_takes_weight_and_gives_no_value():
    s = torch.tensor([[[1.0, 2.0]]], dtype=torch.float64)
    p = R.sink_softmax(s, torch.tensor([0.5], dtype=torch.float64))
    den = math.exp(1) + math.exp(2) + math.exp(0.5)
    assert torch.allclose(p[0, 0], torch.tensor([math.exp(1) / den, math.exp(2) / den], dtype=torch.float64))


def test_oracle_rotation_depends_on_distance_only():
    torch.manual_seed(1)
    a, b = torch.randn(1, 8, dtype=torch.float64), torch.randn(1, 8, dtype=torch.float64)
    rot = lambda x, p: R.rotate_interleaved(x, torch.tensor([p]), 500.0, 8)
    assert torch.allclose((rot(a, 3) * rot(b, 10)).sum(), (rot(a, 40) * rot(b, 47)).sum())
    x = torch.zeros(1, 4, dtype=torch.float64)
    x[0, 0] = 1.0                                      # pair (0, 1) turns by p radians
    x = R.rotate_interleaved(x, torch.tensor([1]), 500.0, 4)
    assert torch.allclose(x[0, :2], torch.tensor([math.cos(1.0), math.sin(1.0)], dtype=torch.float64))
