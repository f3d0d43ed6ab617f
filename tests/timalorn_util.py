"""Small Timalorn configurations for the tests (sizes unlike any trained model's)."""


def attention(heads=4, kv_heads=2, dim=24, window=37, rot_dims=8, base=3000.0, scale=0.3, softcap=6.0, factor=3.0, original=48,
              fast=5.0, slow=0.6, ff=72, weights_of=None):
    e = {"type": "attention",
         "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap,
                   "mask": {"size": window},
                   "rot": {"base": base, "dims": rot_dims,
                           "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}},
         "mlp": {"kind": "dense", "ff": ff} if ff else None}
    return e if weights_of is None else dict(e, weights_of=weights_of)


def memory(heads=3, dim=16, vdim=24, gate_cap=4.0, ff=40, weights_of=None):
    e = {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap},
         "mlp": {"kind": "dense", "ff": ff} if ff else None}
    return e if weights_of is None else dict(e, weights_of=weights_of)


def config(layers, width=80, vocab=131, scale=2.0, eps=3e-5):
    return {"architecture": "Timalorn", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


CONFIGS = {
    # both mixers, with and without a feed-forward, shared tensors of both kinds
    "shared": config([attention(), memory(), attention(weights_of=0), memory(heads=2, dim=24, vdim=16, ff=0),
                      memory(weights_of=1), attention(heads=2, kv_heads=1, window=9, ff=0)]),
    # nothing shared but with a later layer; whole heads turned, no stretching to speak of, a window larger than any
    # prompt, as many key heads as query heads; values wider than keys by far
    "plain": config([memory(heads=2, dim=8, vdim=64, gate_cap=15.0, weights_of=2),
                     attention(heads=3, kv_heads=3, dim=32, rot_dims=32, window=4096, factor=1.0, softcap=30.0, base=10000.0),
                     memory(heads=2, dim=8, vdim=64, gate_cap=15.0)], width=72, vocab=97, scale=1.0),
    # sizes that are no multiple of 8, windows of 1, 2 and 5, the narrowest rotation
    "odd": config([attention(heads=3, kv_heads=1, dim=14, rot_dims=6, window=5, ff=30),
                   attention(heads=2, kv_heads=2, dim=9, rot_dims=2, window=1, ff=0), memory(heads=3, dim=13, vdim=11, ff=22),
                   attention(heads=2, kv_heads=1, dim=10, rot_dims=10, window=2, ff=22)], width=54, vocab=61),
    # tensor-core sized heads
    "wide": config([attention(heads=4, kv_heads=2, dim=48, rot_dims=32, window=96, ff=128, softcap=9.0),
                    memory(heads=4, dim=56, vdim=72, ff=96, gate_cap=8.0),
                    attention(heads=6, kv_heads=1, dim=80, rot_dims=16, window=70, ff=64), memory(heads=2, dim=136, vdim=32, ff=0)],
                   width=160, vocab=203),
}
