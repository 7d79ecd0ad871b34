"""Plain, slow restatement of the Kalonex decoder in PyTorch: one function per mechanism, no cache, no kernels, nothing
shared with the package. Every function takes the whole sequence of ONE request and works in the dtype of its inputs; the
tests run it in float64.

``weights`` is a dict ``name -> tensor`` with the checkpoint's tensor names, ``cfg`` the parsed ``config.json``.
"""
import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def linear(x, w, b=None):
    y = x @ w.t()
    return y if b is None else y + b


def rotate_half(x, pos, base, dims):
    """Rotary positions on the first ``dims`` of the last dimension; dimension i turns with i + dims/2. ``x (T, H, D)``."""
    out = x.clone()
    for i in range(dims // 2):
        a = (pos.to(x.dtype) * base ** (-2.0 * i / dims))[:, None]
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + dims // 2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def window_mask(n, size):
    """(n, n) booleans: query i sees key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < size)


def sink_softmax(s, seen, sink):
    """Softmax of ``s (H, T, T)`` over the seen entries; each head's denominator has one more entry exp(sink)."""
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def attention_core(q, k, v, scale, size, sink):
    """``q (T, H, D)``, ``k (T, G, D)``, ``v (T, G, Dv)`` -> ``(T, H, Dv)``; head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    share = H // k.shape[1]
    head = torch.arange(H) // share
    s = torch.einsum("ihd,jhd->hij", q, k[:, head]) * scale
    return torch.einsum("hij,jhd->ihd", sink_softmax(s, window_mask(T, size), sink), v[:, head])


def attention(h, w, p, m, eps):
    """The mixer; ``w`` by name, ``p`` the prefix of its tensors, ``m`` its entry of the configuration."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (linear(h, w[p + n], w[p + n + ".b"]) for n in "qkv")
    q, k = norm(q, w[p + "q.norm"], eps), norm(k, w[p + "k.norm"], eps)
    pos = torch.arange(T)
    q = rotate_half(q.view(T, H, D), pos, m["rot"]["base"], m["rot"]["dims"])
    k = rotate_half(k.view(T, G, D), pos, m["rot"]["base"], m["rot"]["dims"])
    o = attention_core(q, k, v.view(T, G, Dv), m["scale"], m["mask"]["size"], w[p + "sink"])
    return linear(o.reshape(T, H * Dv), w[p + "o"], w[p + "o.b"])


def gated(h, w, p):
    """Gated feed-forward: down(silu(gate h) * (up h))."""
    return linear(silu(linear(h, w[p + "gate"])) * linear(h, w[p + "up"]), w[p + "down"])


def route(h, w_router, top):
    """(chosen experts, weights), both ``(T, top)``: the largest sigmoid scores, as they are."""
    s = sigmoid(linear(h, w_router))
    order = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return order, torch.gather(s, 1, order)


def experts(h, w, p, mlp):
    """Routed experts (the score multiplies an expert's input) and the expert that runs for every token."""
    chosen, weight = route(h, w[p + "router"], mlp["router"]["top"])
    out = gated(h, w, p + "shared.") if mlp.get("shared") is not None else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weight[t]):
            out[t] = out[t] + gated(s * h[t], w, f"{p}e{e}.")
    return out


def layer(x, w, i, entry, eps):
    x = x + attention(norm(x, w[f"l{i}.norm1"], eps), w, f"l{i}.mix.", entry["mixer"], eps)
    mlp = entry["mlp"]
    if mlp is None:
        return x
    h = norm(x, w[f"l{i}.norm2"], eps)
    return x + (gated(h, w, f"l{i}.mlp.") if mlp["kind"] == "dense" else experts(h, w, f"l{i}.mlp.", mlp))


def enter_pass(x, x0, w, t):
    """What happens once before pass ``t`` over the looped layers."""
    return linear(torch.cat([x, x0], -1), w["loop.in"]) + w["loop.step"][t]


def schedule(cfg):
    """(layer, pass it begins or None) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg["loop"]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, weights, tokens, taps=None, dtype=torch.float64):
    """Logits ``(T, vocab)`` of a whole sequence; ``taps`` collects the residual stream after every layer run."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens)]
    x = x0
    for i, t in schedule(cfg):
        if t is not None:
            x = enter_pass(x, x0, w, t)
        x = layer(x, w, i, cfg["layers"][i], eps)
        if taps is not None:
            taps.append(x)
    return linear(norm(x, w["final.norm"], eps), w["head"]) * cfg["logit_scale"]


# ---------------------------------------------------------------------------------------------------------------------
def shapes(cfg):
    """Names and shapes of a checkpoint."""
    d, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}

    def ff(p, n):
        out.update({p + "gate": (n, d), p + "up": (n, d), p + "down": (d, n)})

    if cfg["loop"]["times"]:
        out.update({"loop.in": (d, 2 * d), "loop.step": (cfg["loop"]["times"], d)})
    for i, e in enumerate(cfg["layers"]):
        m, mlp, p = e["mixer"], e["mlp"], f"l{i}."
        nq, nk, nv, no = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        out[p + "norm1"] = (d,)
        for n, r in (("q", nq), ("k", nk), ("v", nv)):
            out.update({p + f"mix.{n}": (r, d), p + f"mix.{n}.b": (r,)})
        out.update({p + "mix.q.norm": (nq,), p + "mix.k.norm": (nk,), p + "mix.sink": (m["heads"],),
                    p + "mix.o": (d, no), p + "mix.o.b": (d,)})
        if mlp is None:
            continue
        out[p + "norm2"] = (d,)
        if mlp["kind"] == "dense":
            ff(p + "mlp.", mlp["ff"])
        else:
            for j in range(mlp["router"]["experts"]):
                ff(f"{p}mlp.e{j}.", mlp["expert"]["ff"])
            out[p + "mlp.router"] = (mlp["router"]["experts"], d)
            if mlp.get("shared") is not None:
                ff(p + "mlp.shared.", mlp["shared"]["ff"])
    out.update({"final.norm": (d,), "head": (cfg["vocab"], d)})
    return out


def random_model(cfg, seed=0):
    """Random bf16 weights that make every mechanism matter: sinks and biases of the size of the scores and projections,
    gains around one."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(*shape, generator=g)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            t = 1 + 0.3 * t
        elif name == "loop.in":
            t = t / math.sqrt(shape[1]) * 1.4
        elif name.endswith(("mlp.router", ".gate", ".up", ".down")) or (len(shape) == 2 and name not in ("embed", "loop.step")):
            t = t / math.sqrt(shape[1])
        elif name.endswith(".b") or name == "loop.step":
            t = 0.5 * t
        w[name] = t.bfloat16()
    return w
