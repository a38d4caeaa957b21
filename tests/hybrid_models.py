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
