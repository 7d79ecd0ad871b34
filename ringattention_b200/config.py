"""Configuration objects: ``BlockwiseKwargs`` (the reference's ``blockwise_kwargs`` dict, validated),
``MeshConfig`` (dp, fsdp, tp, sp), ``LlamaConfig`` and ``TrainConfig``.

The reference has no config system: it passes a plain dict whose ten keys are positional
parameters of its blockwise functions (ringattention/ringattention_jax.py:99-100, README.md:25-36).
``BlockwiseKwargs.from_any`` accepts that dict verbatim.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Union

import torch

# Remat policies understood by this library. The reference forwards a jax.checkpoint policy
# (ringattention_jax.py:130,334); only the two below have an effect here.
POLICY_NOTHING_SAVEABLE = "nothing_saveable"
POLICY_EVERYTHING_SAVEABLE = "everything_saveable"
# Model-level extension: recompute a layer in the backward pass except its attention, whose output and
# log-sum-exp are kept (0.5 GB per layer at 64K tokens x 4096). Not one of the reference's policies.
POLICY_SAVE_ATTENTION = "save_attention"

_REFERENCE_KEYS = (
    "causal_block_size", "query_chunk_size", "key_chunk_size", "deterministic", "dropout_rng",
    "attn_pdrop", "dtype", "policy", "precision", "prevent_cse",
)
_EXTENSION_KEYS = ("layout",)


def _policy_name(policy: Any) -> str:
    if policy is None:
        return POLICY_NOTHING_SAVEABLE
    if isinstance(policy, str):
        name = policy
    else:  # e.g. a function object named like jax.checkpoint_policies.nothing_saveable
        name = getattr(policy, "__name__", str(policy))
    if "nothing" in name:
        return POLICY_NOTHING_SAVEABLE
    if "everything" in name or "dots" in name or "save" in name:
        return POLICY_EVERYTHING_SAVEABLE
    raise ValueError(f"unknown remat policy {policy!r}")


@dataclass
class BlockwiseKwargs:
    """Validated form of the reference's ``blockwise_kwargs``.

    ``causal_block_size``: ``None`` no causal mask, 1 causal, k>1 block-causal (token i sees j iff
    ``i // k >= j // k``; ringattention_jax.py:301-309). ``query_chunk_size``/``key_chunk_size`` must
    divide the local lengths (ringattention_jax.py:104-108); results do not depend on them.
    Dropout is active iff ``not deterministic and attn_pdrop > 0``; dropped logits are masked before
    the softmax without 1/(1-p) rescaling (ringattention_jax.py:119-123,311-321).
    ``dropout_rng`` is an int seed or a ``torch.Generator`` (a seed is drawn from it).
    ``layout`` is an extension: ``"contiguous"`` (reference behaviour: rank r owns tokens
    ``[r*c, (r+1)*c)``), ``"zigzag"`` (rank r owns chunks r and 2N-1-r of 2N, which balances
    causal work across the ring) or ``"pairs:a0-b0,..."`` (an explicit pairing of the 2N half-chunks, e.g. the one
    ``ops.reference.balanced_pairs`` derives from the document boundaries of a packed batch).
    """

    causal_block_size: Optional[int] = None
    query_chunk_size: int = 128
    key_chunk_size: int = 128
    deterministic: bool = True
    dropout_rng: Any = None
    attn_pdrop: float = 0.0
    dtype: Any = torch.float32
    policy: str = POLICY_NOTHING_SAVEABLE
    precision: Any = None
    prevent_cse: bool = True
    layout: str = "contiguous"

    @classmethod
    def from_any(cls, obj: "BlockwiseKwargs | Mapping[str, Any] | None") -> "BlockwiseKwargs":
        if obj is None:
            return cls()
        if isinstance(obj, cls):
            return obj
        if not isinstance(obj, Mapping):
            raise TypeError("blockwise_kwargs must be a dict or BlockwiseKwargs")
        unknown = set(obj) - set(_REFERENCE_KEYS) - set(_EXTENSION_KEYS)
        if unknown:
            raise KeyError(f"unknown blockwise_kwargs keys: {sorted(unknown)}")
        kw = dict(obj)
        if "policy" in kw:
            kw["policy"] = _policy_name(kw["policy"])
        out = cls(**kw)
        out.validate()
        return out

    def validate(self) -> None:
        if self.causal_block_size is not None and int(self.causal_block_size) < 1:
            raise ValueError("causal_block_size must be None or >= 1")
        if self.query_chunk_size < 1 or self.key_chunk_size < 1:
            raise ValueError("chunk sizes must be positive")
        if not (0.0 <= float(self.attn_pdrop) < 1.0):
            raise ValueError("attn_pdrop must be in [0, 1)")
        if self.layout not in ("contiguous", "zigzag") and not str(self.layout).startswith("pairs:"):
            raise ValueError("layout must be 'contiguous', 'zigzag' or 'pairs:a0-b0,a1-b1,...'")

    @property
    def dropout_active(self) -> bool:
        return (not self.deterministic) and float(self.attn_pdrop) > 0.0

    def seed(self) -> int:
        """64-bit dropout seed derived from ``dropout_rng`` (0 when dropout is inactive)."""
        if not self.dropout_active:
            return 0
        rng = self.dropout_rng
        if rng is None:
            raise ValueError("dropout is active but dropout_rng is None")
        if isinstance(rng, torch.Generator):
            return int(torch.randint(0, 2**62, (1,), generator=rng).item())
        if isinstance(rng, torch.Tensor):
            return int(rng.flatten()[0].item()) & (2**63 - 1)
        return int(rng) & (2**63 - 1)


@dataclass(frozen=True)
class SegmentIds:
    """Per-token segment ids of the queries and of the keys/values of one attention call (the
    reference's ``SegmentIds`` NamedTuple, ringattention_pallas_tpu.py:201-215). Tokens attend only
    to tokens with an equal id."""

    q: Any
    kv: Any


@dataclass(frozen=True)
class BlockSizes:
    """Tile sizes of the fused kernels. The reference exposes eleven tunable TPU tile sizes
    (ringattention_pallas_tpu.py:218-287, default 128 everywhere); the sm_100a kernels are built for
    one tile shape, fixed by the tcgen05 instruction shape and the TMEM budget, so this object is
    informational: ``validate`` only checks that a request is compatible."""

    block_q: int = 256          # query rows per CTA in the forward (two 128-row tiles)
    block_k: int = 128          # key rows per pipeline step
    block_q_bwd: int = 128      # query rows per backward iteration
    block_k_bwd: int = 128      # key rows per backward CTA
    block_b: int = 1

    @classmethod
    def get_default(cls) -> "BlockSizes":
        return cls()

    def validate(self, q_len: int, kv_len: int) -> None:
        if self.block_b != 1:
            raise ValueError("block_b must be 1")
        for name in ("block_q", "block_k", "block_q_bwd", "block_k_bwd"):
            v = getattr(self, name)
            if v % 128:
                raise ValueError(f"{name} must be a multiple of 128")
        if q_len < 1 or kv_len < 1:
            raise ValueError("empty sequence")


@dataclass
class MeshConfig:
    """Sizes of the four mesh axes used in the reference's README (README.md:38-46)."""

    dp: int = 1
    fsdp: int = 1
    tp: int = 1
    sp: int = 1

    AXES = ("dp", "fsdp", "tp", "sp")

    @classmethod
    def parse(cls, text: "str | MeshConfig | None") -> "MeshConfig":
        """Parse ``"1,2,1,4"`` (dp,fsdp,tp,sp) or ``"fsdp=2,sp=4"``."""
        if text is None:
            return cls()
        if isinstance(text, cls):
            return text
        parts = [p.strip() for p in str(text).split(",") if p.strip()]
        if all("=" in p for p in parts):
            kv = {}
            for p in parts:
                k, v = p.split("=")
                if k.strip() not in cls.AXES:
                    raise ValueError(f"unknown mesh axis {k!r}")
                kv[k.strip()] = int(v)
            return cls(**kv)
        if len(parts) != 4:
            raise ValueError("mesh must be 'dp,fsdp,tp,sp' or 'axis=size,...'")
        return cls(*[int(p) for p in parts])

    @property
    def world_size(self) -> int:
        return self.dp * self.fsdp * self.tp * self.sp

    def shape(self) -> tuple[int, int, int, int]:
        return (self.dp, self.fsdp, self.tp, self.sp)

    def describe(self) -> str:
        return "x".join(f"{a}{getattr(self, a)}" for a in self.AXES if getattr(self, a) > 1) or "single"


@dataclass
class LlamaConfig:
    """LLaMA-style decoder. Defaults are the 7B shape."""

    vocab_size: int = 32000
    d_model: int = 4096
    n_layers: int = 32
    n_heads: int = 32
    d_ff: int = 11008
    rms_eps: float = 1e-6
    rope_theta: float = 10000.0
    init_std: float = 0.02
    max_seq_len: int = 1 << 20
    # attention / ffn chunking
    query_chunk_size: int = 2048
    key_chunk_size: int = 2048
    ffn_chunk_size: int = 8192
    loss_chunk_size: int = 8192
    causal_block_size: int = 1
    remat: str = POLICY_NOTHING_SAVEABLE
    layout: str = "contiguous"

    @property
    def head_dim(self) -> int:
        return self.d_model // self.n_heads

    def n_params(self, include_embedding: bool = True) -> int:
        per_layer = 4 * self.d_model * self.d_model + 3 * self.d_model * self.d_ff + 2 * self.d_model
        n = self.n_layers * per_layer + self.d_model + self.vocab_size * self.d_model
        if include_embedding:
            n += self.vocab_size * self.d_model
        return n

    @classmethod
    def named(cls, name: str, **over) -> "LlamaConfig":
        presets = {
            "llama-7b": dict(),
            "llama-1b": dict(d_model=2048, n_layers=16, n_heads=16, d_ff=5504),
            "llama-tiny": dict(vocab_size=1024, d_model=256, n_layers=2, n_heads=2, d_ff=512,
                               query_chunk_size=128, key_chunk_size=128, ffn_chunk_size=256,
                               loss_chunk_size=256),
            "llama-small": dict(vocab_size=4096, d_model=512, n_layers=2, n_heads=4, d_ff=1536,
                                query_chunk_size=256, key_chunk_size=256, ffn_chunk_size=512,
                                loss_chunk_size=512),
        }
        if name not in presets:
            raise KeyError(f"unknown model {name!r}; have {sorted(presets)}")
        kw = dict(presets[name])
        kw.update(over)
        return cls(**kw)


@dataclass(frozen=True)
class RotaryConfig:
    """Rotary positions on the first ``dims`` dimensions of a vector, frequencies ``base ** (-2i / dims)``. The mixer that
    uses it fixes the pairs: (2i, 2i + 1) in latent attention, (i, i + dims / 2) in windowed attention."""

    base: float
    dims: int

    def inv_freq(self) -> list:
        return [float(self.base) ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]


@dataclass(frozen=True)
class LatentAttentionConfig:
    """Latent attention: per token a ``kv_rank`` latent and one rotated key part of ``rot_dim`` are cached; heads have
    ``dim`` unrotated and ``rot_dim`` rotated query/key dimensions and ``vdim`` value dimensions."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: RotaryConfig

    def __post_init__(self):
        if self.rot.dims % 2 or not 0 <= self.rot.dims <= self.rot_dim:
            raise ValueError("rotary dims must be even and at most rot_dim")


@dataclass(frozen=True)
class GatedDeltaConfig:
    """Gated delta rule with short convolutions over ``conv`` tokens: ``heads`` states of ``dim`` x ``vdim``, value head h
    uses q/k head ``h // (heads // kv_heads)``."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")


@dataclass(frozen=True)
class WindowAttentionConfig:
    """Attention of ``heads`` query heads over ``kv_heads`` key/value heads (query head h reads head ``h // (heads //
    kv_heads)``) with biases in the projections, RMS norms over the whole query and key projections, rotary positions on
    the first dimensions of a head and a learned sink per head. A query sees itself and the ``window - 1`` tokens before it
    (None: everything before it)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotaryConfig
    window: Optional[int] = None

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if self.rot.dims % 2 or not 0 <= self.rot.dims <= self.dim:
            raise ValueError("rotary dims must be even and at most dim")
        if self.window is not None and self.window < 1:
            raise ValueError("a window holds at least the token itself")


@dataclass(frozen=True)
class DenseConfig:
    """Feed-forward: ``down(relu(up x)^2)``, or with ``gated`` ``down(silu(gate x) * (up x))``."""

    ff: int
    gated: bool = False


@dataclass(frozen=True)
class MoEConfig:
    """Routed experts: of ``experts`` gated feed-forwards of width ``ff`` a token uses the ``top`` with the largest sigmoid
    scores; the score multiplies the expert's input. A ``shared_ff`` wide one runs for every token (None: there is none)."""

    experts: int
    top: int
    ff: int
    shared_ff: Optional[int] = None

    def __post_init__(self):
        if not 1 <= self.top <= self.experts:
            raise ValueError("a token uses at least one and at most all experts")


MixerConfig = Union[LatentAttentionConfig, GatedDeltaConfig, WindowAttentionConfig]


@dataclass(frozen=True)
class LoopConfig:
    """Layers ``start .. stop - 1`` run ``times`` times in a row with the same tensors; every pass has caches of its own."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerConfig:
    """One decoder layer: a mixer, an optional feed-forward and, when the layer has no tensors of its own, the index of
    the layer whose tensors it uses (its cache or state is its own all the same)."""

    mixer: MixerConfig
    mlp: Union[DenseConfig, MoEConfig, None] = None
    weights_of: Optional[int] = None


@dataclass(frozen=True)
class Design:
    """What an architecture fixes for all its models."""

    norm_gain_offset: float   # 1: norm gains are stored around zero
    parallel: bool            # mixer and feed-forward read the same stream and are added together; else one after the other
    gated: bool               # dense feed-forwards are gated
    mixers: tuple             # mixer types of a config.json


DESIGNS = {
    "Dafelorn": Design(norm_gain_offset=1.0, parallel=True, gated=False, mixers=("latent_attention", "delta")),
    "Kalonex": Design(norm_gain_offset=0.0, parallel=False, gated=True, mixers=("attention",)),
}


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``enter`` is the number of the pass that begins with it, None inside a pass or outside
    the loop."""

    layer: int
    enter: Optional[int] = None


@dataclass(frozen=True)
class HybridConfig:
    """Decoder whose layers are listed one by one, each with a mixer and a feed-forward of its own kind. ``architecture``
    names the design: in Dafelorn mixer and feed-forward of a layer read the same residual stream and are added to it
    together; in Kalonex they follow one another, and some layers run several times (``loop``)."""

    vocab_size: int
    d_model: int
    layers: tuple
    rms_eps: float
    architecture: str = "Dafelorn"
    loop: Optional[LoopConfig] = None
    logit_scale: float = 1.0

    def __post_init__(self):
        l = self.loop
        if l is not None and not (0 <= l.start < l.stop <= len(self.layers) and l.times >= 1):
            raise ValueError("the loop does not lie within the layers")

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    @property
    def norm_gain_offset(self) -> float:
        return self.design.norm_gain_offset

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> tuple:
        """The layer runs in the order of execution; every run has a cache or state of its own."""
        l = self.loop
        if l is None:
            return tuple(LayerRun(i) for i in range(self.n_layers))
        looped = [LayerRun(i, t if i == l.start else None) for t in range(l.times) for i in range(l.start, l.stop)]
        return tuple([LayerRun(i) for i in range(l.start)] + looped + [LayerRun(i) for i in range(l.stop, self.n_layers)])

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ValueError("weights_of goes round in a circle")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def n_params(self, include_embedding: bool = True) -> int:
        d = self.d_model
        n = self.vocab_size * d * (2 if include_embedding else 1) + (2 * d * d if self.loop is not None else 0)
        for i, layer in enumerate(self.layers):
            if self.owner(i) != i:
                continue
            m, f = layer.mixer, layer.mlp
            if isinstance(m, LatentAttentionConfig):
                n += d * (m.heads * (m.dim + m.rot_dim) + m.kv_rank + m.rot_dim + m.heads + m.heads * m.vdim)
                n += m.kv_rank * m.heads * (m.dim + m.vdim)
            elif isinstance(m, WindowAttentionConfig):
                n += d * (m.heads + m.kv_heads) * (m.dim + m.vdim)
            else:
                n += d * (2 * m.kv_heads * m.dim + 3 * m.heads * m.vdim + 2 * m.heads)
            if isinstance(f, MoEConfig):
                n += d * (f.experts + 3 * f.experts * f.ff + 3 * (f.shared_ff or 0))
            elif f is not None:
                n += (3 if f.gated else 2) * d * f.ff
        return n

    def cache_bytes(self, context: int, element_bytes: int = 2, max_step: int = 1 << 30) -> int:
        """Bytes that the caches of one sequence of ``context`` tokens take (recurrent states aside)."""
        n = 0
        for r in self.runs:
            m = self.layers[r.layer].mixer
            if isinstance(m, LatentAttentionConfig):
                n += context * (m.kv_rank + m.rot_dim)
            elif isinstance(m, WindowAttentionConfig):
                rows = context if m.window is None else min(context, m.window + min(max_step, context))
                n += rows * m.kv_heads * (m.dim + m.vdim)
        return n * element_bytes

    @staticmethod
    def _mixer_from_dict(kind: str, m: Mapping[str, Any]) -> MixerConfig:
        if kind == "latent_attention":
            return LatentAttentionConfig(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
                                         kv_rank=m["kv_rank"], scale=m["scale"],
                                         rot=RotaryConfig(base=m["rot"]["base"], dims=m["rot"]["dims"]))
        if kind == "attention":
            mask = m.get("mask")
            return WindowAttentionConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                                         scale=m["scale"], rot=RotaryConfig(base=m["rot"]["base"], dims=m["rot"]["dims"]),
                                         window=None if mask is None else mask["size"])
        return GatedDeltaConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=m["conv"])

    @classmethod
    def from_dict(cls, c: Mapping[str, Any]) -> "HybridConfig":
        """Parse a ``config.json`` of one of the designs."""
        arch = c.get("architecture", "Dafelorn")
        design = DESIGNS[arch]
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] not in design.mixers:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            mixer = cls._mixer_from_dict(e["type"], e["mixer"])
            f = e.get("mlp")
            if f is None:
                mlp = None
            elif f["kind"] == "dense":
                mlp = DenseConfig(ff=f["ff"], gated=design.gated)
            elif f["kind"] == "moe" and design.gated:
                shared = f.get("shared")
                mlp = MoEConfig(experts=f["router"]["experts"], top=f["router"]["top"], ff=f["expert"]["ff"],
                                shared_ff=None if shared is None else shared["ff"])
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            w = e.get("weights_of")
            if w is not None and not 0 <= w < len(c["layers"]):
                raise ValueError(f"layer {i}: weights_of {w} is not a layer")
            layers.append(LayerConfig(mixer, mlp, w))
        loop = c.get("loop")
        out = cls(vocab_size=c["vocab"], d_model=c["width"], layers=tuple(layers), rms_eps=c["norm"]["eps"],
                  architecture=arch, logit_scale=float(c.get("logit_scale", 1.0)),
                  loop=None if loop is None else LoopConfig(loop["start"], loop["stop"], loop["times"]))
        for i in range(out.n_layers):
            j = out.owner(i)
            if (out.layers[i].mixer, out.layers[i].mlp) != (out.layers[j].mixer, out.layers[j].mlp):
                raise ValueError(f"layer {i} uses the tensors of layer {j} but has other sizes")
        return out

    @classmethod
    def named(cls, name: str, **over) -> "HybridConfig":
        """Presets of LLaMA-like sizes."""
        def dafelorn(n, heads, dim, rot, rank, ff, dk):
            """Three delta layers to one latent-attention layer."""
            lat = LatentAttentionConfig(heads=heads, dim=dim, rot_dim=rot, vdim=dim, kv_rank=rank,
                                        scale=(dim + rot) ** -0.5, rot=RotaryConfig(10000.0, rot))
            dl = GatedDeltaConfig(heads=heads, kv_heads=heads // 2, dim=dk, vdim=dk, conv=4)
            return dict(layers=tuple(LayerConfig(lat if i % 4 == 3 else dl, DenseConfig(ff)) for i in range(n)))

        def kalonex(n, heads, kv_heads, dim, window, ff, experts, top, expert_ff, shared_ff):
            """``n`` layer runs: a dense and a routed layer, then (n - 2) / 2 passes over two more of them. The routed
            layers' active feed-forward (top experts and the shared one) is as wide as the dense one."""
            if n < 4 or n % 2:
                raise ValueError("this preset has an even number of layer runs, at least four")
            at = WindowAttentionConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5,
                                       rot=RotaryConfig(10000.0, dim // 2), window=window)
            dense, moe = DenseConfig(ff, gated=True), MoEConfig(experts, top, expert_ff, shared_ff)
            return dict(layers=tuple(LayerConfig(at, f) for f in (dense, moe, dense, moe)),
                        loop=LoopConfig(2, 4, (n - 2) // 2))

        presets = {
            "dafelorn-7b": dict(vocab_size=32000, d_model=4096, rms_eps=1e-6,
                                stack=dict(n=32, heads=32, dim=128, rot=64, rank=512, ff=16512, dk=128)),
            "dafelorn-1b": dict(vocab_size=32000, d_model=2048, rms_eps=1e-6,
                                stack=dict(n=16, heads=16, dim=128, rot=64, rank=512, ff=8256, dk=128)),
            "dafelorn-tiny": dict(vocab_size=1024, d_model=256, rms_eps=1e-6,
                                  stack=dict(n=4, heads=2, dim=64, rot=32, rank=64, ff=768, dk=64)),
            "kalonex-7b": dict(vocab_size=32000, d_model=4096, rms_eps=1e-6,
                               stack=dict(n=32, heads=32, kv_heads=8, dim=128, window=4096, ff=11008, experts=64, top=8,
                                          expert_ff=1152, shared_ff=1792)),
            "kalonex-1b": dict(vocab_size=32000, d_model=2048, rms_eps=1e-6,
                               stack=dict(n=16, heads=16, kv_heads=4, dim=128, window=2048, ff=5504, experts=32, top=4,
                                          expert_ff=1024, shared_ff=1408)),
            "kalonex-tiny": dict(vocab_size=1024, d_model=256, rms_eps=1e-6,
                                 stack=dict(n=4, heads=4, kv_heads=2, dim=64, window=128, ff=512, experts=8, top=2,
                                            expert_ff=128, shared_ff=256)),
        }
        if name not in presets:
            raise KeyError(f"unknown model {name!r}; have {sorted(presets)}")
        kw = dict(presets[name])
        arch = name.split("-")[0].capitalize()
        st = dict(kw.pop("stack"))
        if "n_layers" in over:
            st["n"] = over.pop("n_layers")
        kw.update({"dafelorn": dafelorn, "kalonex": kalonex}[name.split("-")[0]](**st), architecture=arch)
        kw.update(over)
        return cls(**kw)


@dataclass
class TrainConfig:
    model: str = "llama-7b"
    mesh: str = "1,1,1,1"
    seq_len: int = 65536          # global sequence length
    global_batch: int = 1
    lr: float = 1e-4
    weight_decay: float = 0.1
    beta1: float = 0.9
    beta2: float = 0.95
    eps: float = 1e-8
    grad_clip: float = 1.0
    steps: int = 10
    seed: int = 0
    packed_mean_doc_len: int = 0  # >0: packed documents with geometric lengths (segment ids)
    balance_documents: bool = True  # packed documents on a ring: pair the half-chunks by their attention work
    zero1: bool = True            # shard fp32 master weights and AdamW moments over the sp/dp replicas
    log_every: int = 1
    ckpt_dir: Optional[str] = None
    ckpt_every: int = 0
    resume: bool = False

    def asdict(self) -> dict:
        return dataclasses.asdict(self)
