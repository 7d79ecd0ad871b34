"""Plain, slow restatement of the Dafelorn decoder in PyTorch: one function per mechanism, no cache, no kernels,
nothing shared with the package. Every function takes the whole sequence (or explicit state) of ONE request and works
in the dtype of its inputs; the tests run it in float64.

``weights`` is a dict ``name -> tensor`` with the checkpoint's tensor names, ``cfg`` the parsed ``config.json``.
"""
import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def silu(x):
    return x / (1 + torch.exp(-x))


def relu_squared(x):
    return torch.where(x > 0, x * x, torch.zeros_like(x))


def softplus(x):
    return torch.where(x > 0, x, torch.zeros_like(x)) + torch.log1p(torch.exp(-x.abs()))


def rotate_interleaved(x, pos, base, dims):
    """Rotary positions on the first ``dims`` of the last dimension; pairs are (2i, 2i + 1). ``x (T, ..., D)``."""
    out = x.clone()
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        a = pos.to(x.dtype) * f
        a = a.reshape([-1] + [1] * (x.dim() - 2))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def causal_conv(x, w):
    """``x (T, C)``, ``w (C, taps)``; the last tap multiplies the current row, rows before the start are zero."""
    T, C = x.shape
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j                                  # how many tokens ago this tap looks
        if back < T:
            out[back:] += x[:T - back] * w[:, j]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def gated_delta_scan(q, k, v, g, beta, state=None):
    """``q, k (T, H, dk)``, ``v (T, H, dv)``, ``g, beta (T, H)``: decay, read with the key, write, read with the query."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out, S


def delta_mixer(h, W, m, eps):
    """``W(name)`` returns the mixer's tensor."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ W(n).t(), W(n + ".conv"))) for n in ("q", "k", "v"))
    rep = H // G
    q = (unit(q.view(T, G, dk)) * dk ** -0.5).repeat_interleave(rep, dim=1)
    k = unit(k.view(T, G, dk)).repeat_interleave(rep, dim=1)
    v = v.view(T, H, dv)
    beta = 1 / (1 + torch.exp(-(h @ W("b").t())))
    g = torch.exp(-torch.exp(W("A_log")) * softplus(h @ W("a").t() + W("dt_bias")))
    o, _ = gated_delta_scan(q, k, v, g, beta)
    o = rms(o, eps) * W("norm") * silu((h @ W("g").t()).view(T, H, dv))
    return o.reshape(T, H * dv) @ W("o").t()


def sink_softmax(scores, sink):
    """``scores (H, Tq, Tk)`` with -inf where hidden, ``sink (H)``: one more entry in the denominator."""
    s = sink[:, None, None].expand(scores.shape[0], scores.shape[1], 1)
    full = torch.cat([scores, s], dim=-1)
    full = full - full.amax(-1, keepdim=True)
    e = torch.exp(full)
    return (e / e.sum(-1, keepdim=True))[..., :-1]


def latent_mixer(h, W, m, eps):
    T = h.shape[0]
    H, dn, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ W("q").t()).view(T, H, dn + dr)
    kv = h @ W("dkv").t()
    c = rms(kv[:, :r], eps) * W("dkv.norm")
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    k_rot = rotate_interleaved(kv[:, r:], pos, base, dims)
    q_rot = rotate_interleaved(q[..., dn:], pos, base, dims)
    k_un = (c @ W("uk").t()).view(T, H, dn)
    val = (c @ W("uv").t()).view(T, H, dv)
    s = torch.einsum("ihd,jhd->hij", q[..., :dn], k_un) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    s = s * m["scale"]
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)
    p = sink_softmax(s.masked_fill(hidden, -math.inf), W("sink"))
    o = torch.einsum("hij,jhd->ihd", p, val)
    gate = 1 / (1 + torch.exp(-(h @ W("g").t())))
    return (o * gate[..., None]).reshape(T, H * dv) @ W("o").t()


def forward(cfg, weights, tokens, dtype=torch.float64, taps=None):
    """Logits ``(T, vocab)`` of one request; ``taps`` (a list) collects the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        mix = {"delta": delta_mixer, "latent_attention": latent_mixer}[layer["type"]]
        y = mix(zero_centred_norm(x, w[p + "norm1"], eps), lambda n: w[p + "mix." + n], layer["mixer"], eps)
        if layer.get("mlp") is not None:
            h2 = zero_centred_norm(x, w[p + "norm2"], eps)
            y = y + relu_squared(h2 @ w[p + "mlp.up"].t()) @ w[p + "mlp.down"].t()
        x = x + y
        if taps is not None:
            taps.append(x.clone())
    return zero_centred_norm(x, w["final.norm"], eps) @ w["head"].t()


def random_model(cfg, seed=0, scale=1.0):
    """Random bf16 weights for a config dict, with magnitudes at which every mechanism matters."""
    g = torch.Generator().manual_seed(seed)
    d, V = cfg["width"], cfg["vocab"]
    w = {}

    def lin(name, n, k, gain=1.0):
        w[name] = (torch.randn(n, k, generator=g) * (gain * scale / math.sqrt(k))).bfloat16()

    def vec(name, n, mean=0.0, std=0.2):
        w[name] = (mean + std * torch.randn(n, generator=g)).bfloat16()

    w["embed"] = torch.randn(V, d, generator=g).bfloat16()
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", d)
        H = m["heads"]
        if layer["type"] == "delta":
            G, dk, dv = m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                lin(p + "mix." + n, rows, d)
                w[p + f"mix.{n}.conv"] = (torch.randn(rows, m["conv"], generator=g) / math.sqrt(m["conv"])).bfloat16()
            lin(p + "mix.b", H, d)
            lin(p + "mix.a", H, d)
            vec(p + "mix.A_log", H, -1.0, 1.0)
            vec(p + "mix.dt_bias", H, -2.0, 1.0)
            vec(p + "mix.norm", dv, 1.0)
            lin(p + "mix.g", H * dv, d)
            lin(p + "mix.o", d, H * dv)
        else:
            dn, dr, dv, r = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            lin(p + "mix.q", H * (dn + dr), d, 2.0)
            lin(p + "mix.dkv", r + dr, d, 1.5)
            vec(p + "mix.dkv.norm", r, 1.0)
            lin(p + "mix.uk", H * dn, r, 1.5)
            lin(p + "mix.uv", H * dv, r)
            vec(p + "mix.sink", H, 0.5, 1.0)
            lin(p + "mix.g", H, d)
            lin(p + "mix.o", d, H * dv)
        if layer.get("mlp") is not None:
            F = layer["mlp"]["ff"]
            vec(p + "norm2", d)
            lin(p + "mlp.up", F, d)
            lin(p + "mlp.down", d, F)
    vec("final.norm", d)
    lin("head", V, d)
    return w
