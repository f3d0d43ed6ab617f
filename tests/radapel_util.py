"""Small Radapel configurations for the tests (sizes unlike any trained model's)."""


def attention(heads=4, kv_heads=2, dim=24, vdim=16, chunk=40, bias_max=21, scale=0.2, ff=72, limit=1.1, mlp=True):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
                      "mask": {"size": chunk}},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if mlp else None}


def latent(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=56, base=5000.0, scale=0.18, ff=56, limit=2.0, mlp=True):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if mlp else None}


def mamba(heads=4, vdim=24, state=16, groups=2, conv=3, norm_groups=4, mlp=False, ff=40, limit=0.7):
    return {"type": "mamba2",
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                      "norm_groups": norm_groups},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if mlp else None}


def config(layers, width=80, vocab=131, loop=None, scale=2.0, eps=3e-5):
    d = {"architecture": "Radapel", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
         "width": width}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CONFIGS = {
    # every mixer, with and without a feed-forward, a loop over the middle
    "looped": config([attention(), latent(), mamba(), attention(heads=2, kv_heads=1, chunk=24, mlp=False), mamba(mlp=True)],
                     loop=(1, 4, 3)),
    # no loop; one group, one norm group, two taps, a chunk larger than any test prompt, multi-query attention
    "plain": config([mamba(heads=2, vdim=40, groups=1, conv=2, norm_groups=1), latent(heads=5, rot_dim=16, kv_rank=24, mlp=False),
                     attention(heads=3, kv_heads=3, dim=16, vdim=32, chunk=4096, bias_max=90)], width=72, vocab=97),
    # the loop is the whole model, run once; tiny chunks; sizes that are no multiple of 8
    "odd": config([attention(heads=3, kv_heads=1, dim=13, vdim=11, chunk=5, bias_max=7, ff=30),
                   latent(heads=2, dim=9, rot_dim=6, vdim=7, kv_rank=19, ff=22),
                   mamba(heads=3, vdim=10, state=6, groups=3, conv=5, norm_groups=3)], width=54, vocab=61, loop=(0, 3, 1)),
    # tensor-core sized heads
    "wide": config([attention(heads=4, kv_heads=2, dim=64, vdim=80, chunk=96, bias_max=80, ff=128),
                    latent(heads=4, dim=48, rot_dim=32, vdim=64, kv_rank=72, ff=128),
                    mamba(heads=4, vdim=64, state=48, groups=1, conv=4, norm_groups=2)], width=160, vocab=203, loop=(1, 3, 2)),
}
