"""Small configurations of the Kalonex decoder for tests: sizes that differ from one another, odd ones among them."""


def layer(heads, kv_heads, dim, vdim, window, rot, scale, mlp, base=10000.0):
    return {"type": "attention", "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=window),
                          rot=dict(base=base, dims=rot))}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": dict(experts=experts, top=top), "expert": dict(ff=ff)}
    return m if shared is None else {**m, "shared": dict(ff=shared)}


def model(vocab, width, layers, loop, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Kalonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "loop": dict(zip(("start", "stop", "times"), loop)), "logit_scale": logit_scale}


# nothing is a multiple of 16, a layer without a feed-forward, the loop starts with the first layer
ODD = model(331, 108, [
    layer(6, 2, 20, 28, 5, 6, 0.3, dense(90), base=300.0),
    layer(3, 3, 12, 20, 33, 12, 0.4, moe(5, 5, 36, shared=20)),
    layer(4, 1, 28, 12, 70, 0, 0.2, None),
], loop=(0, 2, 2), eps=1e-4, logit_scale=0.3)

# sizes of the tensor-core kernels; groups of 2, 6 and 20 heads; the loop ends with the last layer
FUSED = model(264, 192, [
    layer(4, 2, 128, 64, 130, 64, 0.09, dense(200)),
    layer(6, 1, 64, 128, 64, 64, 0.12, moe(3, 3, 72, shared=136), base=777.0),
    layer(40, 2, 48, 40, 200, 16, 0.15, dense(104)),
    layer(9, 3, 32, 72, 128, 16, 0.2, moe(2, 2, 40)),
], loop=(1, 4, 2), eps=1e-6, logit_scale=1.7)

# experts that are chosen: more than a warp of them, several per token, one per token
ROUTED = model(320, 128, [
    layer(4, 4, 32, 32, 40, 32, 0.18, moe(37, 4, 48, shared=64)),
    layer(8, 2, 16, 24, 17, 8, 0.25, moe(12, 1, 56, shared=8)),
    layer(2, 1, 40, 40, 64, 16, 0.2, moe(6, 2, 200)),
], loop=(1, 2, 3), logit_scale=2.5)

# one of everything: head, expert, pass, and a window that holds the token itself only; heads wider than 128 elsewhere
ONES = model(64, 64, [
    layer(1, 1, 8, 8, 1, 2, 0.5, moe(1, 1, 8)),
    layer(2, 1, 160, 136, 50, 80, 0.08, dense(48)),
    layer(1, 1, 16, 264, 1000, 16, 0.3, dense(8), base=50.0),
], loop=(0, 3, 1), eps=1e-3)

CONFIGS = {"odd": ODD, "fused": FUSED, "routed": ROUTED, "ones": ONES}
