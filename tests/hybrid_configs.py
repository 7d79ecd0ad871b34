"""Small configurations of the hybrid decoder for tests: sizes that differ from one another, odd ones among them."""


def delta(heads, kv_heads, dim, vdim, conv, ff=None, **more):
    return {"type": "delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}, **more}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, ff=None, **more):
    return {"type": "latent_attention",
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                          rot=dict(base=base, dims=rot_dim)),
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}, **more}


def model(vocab, width, layers, eps=1e-5):
    return {"architecture": "Dafelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# nothing is a multiple of 16, layers without a feed-forward, weights used by later layers
TWO_KINDS = model(331, 108, [
    delta(6, 2, 24, 40, 4, ff=90),
    latent(3, 20, 6, 28, 52, 0.3, base=300.0, ff=70),
    delta(3, 3, 12, 20, 2),
    latent(3, 20, 6, 28, 52, 0.3, base=300.0, ff=70, weights_of=1),
    delta(6, 2, 24, 40, 4, ff=90, weights_of=0),
], eps=1e-4)

# sizes of the fused kernels: head parts in multiples of 64, key dimension 128
WIDE = model(256, 256, [
    delta(4, 2, 128, 128, 4, ff=512),
    latent(4, 128, 64, 128, 256, 0.08, ff=384),
    latent(2, 64, 32, 128, 128, 0.11, base=777.0, ff=256),
], eps=1e-6)

# one head, one tap, state wider than long, and one key head for all value heads
ONES = model(64, 64, [
    latent(1, 16, 2, 8, 24, 0.5, ff=48),
    delta(5, 1, 8, 72, 1, ff=40),
    delta(1, 1, 96, 16, 5, ff=32),
    latent(7, 8, 8, 16, 8, 0.9),
], eps=1e-3)

CONFIGS = {"two_kinds": TWO_KINDS, "wide": WIDE, "ones": ONES}
