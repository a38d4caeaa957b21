"""Small hybrid configurations for the tests, as the dictionaries their ``config.json`` would hold.  Sizes are chosen to be
awkward: widths and head sizes that are no multiples of 8 or 16, unequal heads, a layer without feed-forward."""


def latent(heads=3, dim=20, rot=6, rank=36, vdim=28, window=21, scale=0.19, base=3000.0, ff=92):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "kv_rank": rank, "vdim": vdim, "scale": scale,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot}}}


def hgrn2(heads=2, dim=22, vdim=18, ff=75):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def wkv(heads=3, dim=18, ff=60):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def design(layers, vocab=203, width=76, eps=3e-5, mult=0.45):
    return {"architecture": "Nikelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


def small_design():
    return design([wkv(), latent(), hgrn2(ff=0), latent(heads=1, dim=16, rot=2, rank=16, vdim=8, window=5, ff=40), hgrn2(heads=1, dim=5, vdim=7),
                   wkv(heads=1, dim=40, ff=0)])


def aligned_design():
    """Sizes near a real model's proportions, still small: several tiles of the tensor-core kernels."""
    return design([latent(heads=20, dim=64, rot=32, rank=160, vdim=48, window=150, scale=0.1, ff=512), hgrn2(heads=2, dim=128, vdim=96, ff=256),
                   wkv(heads=4, dim=64, ff=384), hgrn2(heads=3, dim=80, vdim=64, ff=0)], vocab=520, width=256, eps=1e-6, mult=0.8)


def single_layer(layer):
    return design([layer], vocab=97, width=68)


# -- Naselorn -------------------------------------------------------------------------------------------------------------
def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, top=2, ff=28, shared=36):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared}}


def lightning(heads=3, dim=20, vdim=14, decay=None, mlp=None):
    return {"type": "lightning", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay or [1 - 0.7 * 0.3 ** h for h in range(heads)])}}


def parallel(heads=4, kv_heads=2, dim=12, vdim=20, chunk=19, scale=0.3, width=42, blocks=3, conv=3, left=0.8, right=0.55, mlp=None):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk}},
                      "right": {"width": width, "blocks": blocks, "conv": conv}, "left_scale": left, "right_scale": right}}


def naselorn(layers, vocab=211, width=84, eps=2e-5, scale=5.0):
    return {"architecture": "Naselorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


def small_naselorn():
    return naselorn([parallel(mlp=moe()), lightning(mlp=dense(50)), lightning(heads=1, dim=7, vdim=33), parallel(heads=2, kv_heads=2, dim=64, vdim=24,
                     chunk=32, width=40, blocks=1, conv=5, left=1.3, right=0.2, mlp=dense()), lightning(heads=2, dim=24, vdim=8, mlp=moe(5, 1, 16, 20))])


def aligned_naselorn():
    """Sizes near a real model's proportions, still small: several tiles of the tensor-core kernels."""
    return naselorn([lightning(heads=3, dim=128, vdim=72, mlp=dense(304)), parallel(heads=6, kv_heads=2, dim=128, vdim=104, chunk=150, scale=0.09,
                     width=384, blocks=6, conv=4, mlp=moe(12, 4, 96, 144)), lightning(heads=5, dim=48, vdim=80, mlp=moe(9, 2, 80, 64)),
                     parallel(heads=4, kv_heads=1, dim=64, vdim=64, chunk=129, scale=0.125, width=96, blocks=4, conv=2)], vocab=536, width=320, eps=1e-6)
