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


# -- Gaborax --------------------------------------------------------------------------------------------------------------
def relu2_moe(experts=5, identity=3, top=2, ff=28, shared=36):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def gated_heads(heads=4, kv_heads=2, dim=20, vdim=12, rot=12, base=700.0, scale=0.3, kv_from=None, mlp=None, scaling=None):
    """Rotate-half attention with a gate per head."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "scale": scale}
    if scaling:
        m["rot"]["scaling"] = scaling
    return {"type": "attention", "mlp": mlp, "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}


def yarn(factor=3.0, original=64, fast=12.0, slow=0.8):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def capped(heads=3, kv_heads=3, dim=14, vdim=22, rot=10, base=300.0, scale=0.4, softcap=6.0, scaling=yarn(), kv_from=None, mlp=None):
    """Attention with neighbouring pairs, biases and squashed scores."""
    e = gated_heads(heads, kv_heads, dim, vdim, rot, base, scale, kv_from, mlp, scaling)
    e["mixer"]["softcap"] = softcap
    return {**e, "type": "attention_2"}


def gaborax(layers, vocab=199, width=92, eps=4e-5):
    return {"architecture": "Gaborax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def small_gaborax():
    return gaborax([capped(mlp=relu2_moe()), gated_heads(mlp=relu2_moe(3, 0, 1, 16, 20)), gated_heads(heads=6, mlp=relu2_moe(2, 5, 4, 7, 33), kv_from=1),
                    capped(heads=2, kv_heads=1, dim=64, vdim=40, rot=64, softcap=3.0), gated_heads(kv_from=1, scale=0.11, base=50.0),
                    capped(heads=4, kv_heads=1, dim=64, vdim=40, rot=24, kv_from=3, scaling=None, mlp=relu2_moe(4, 1, 3, 24, 8))])


def aligned_gaborax():
    """Sizes near a real model's proportions, still small: several tiles of the tensor-core kernels."""
    return gaborax([gated_heads(heads=6, kv_heads=2, dim=128, vdim=104, rot=96, scale=0.09, mlp=relu2_moe(12, 4, 4, 96, 144)),
                    capped(heads=4, kv_heads=4, dim=64, vdim=64, rot=64, scale=0.125, softcap=15.0, mlp=relu2_moe(9, 2, 2, 80, 64)),
                    gated_heads(heads=6, kv_heads=2, dim=128, vdim=104, rot=96, scale=0.09, kv_from=0, mlp=relu2_moe(6, 1, 3, 64, 80)),
                    capped(heads=8, kv_heads=1, dim=80, vdim=96, rot=48, scale=0.11, softcap=30.0)], vocab=528, width=304, eps=1e-6)


# -- Gaparax --------------------------------------------------------------------------------------------------------------
def relu2_dense(ff=70):
    return {"kind": "dense", "ff": ff}


def group_moe(experts=6, groups=3, keep=2, top=3, ff=28, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}}


def sigmoid_heads(heads=4, kv_heads=2, dim=20, vdim=12, chunk=23, scale=0.3, softcap=6.0, bias_max=15, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                                                      "bias_max": bias_max, "mask": {"size": chunk}}}


def sink_latent(heads=3, dim=20, rot=6, rank=36, vdim=28, scale=0.19, base=300.0, scaling=yarn(), mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "kv_rank": rank, "vdim": vdim, "scale": scale,
                                                             "rot": {"base": base, "dims": rot, "scaling": scaling}}}


def gaparax(layers, vocab=193, width=84, eps=4e-5, streams=3):
    return {"architecture": "Gaparax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers}


def small_gaparax():
    return gaparax([sigmoid_heads(mlp=group_moe()), sink_latent(mlp=relu2_dense()), sigmoid_heads(heads=3, kv_heads=3, dim=7, vdim=33, chunk=50, softcap=2.0,
                    bias_max=120, mlp=relu2_dense(33)), sink_latent(heads=1, dim=16, rot=2, rank=16, vdim=8, scaling=None), sigmoid_heads(heads=5, kv_heads=1, dim=64,
                    vdim=40, chunk=7, bias_max=4), sink_latent(heads=4, dim=64, rot=64, rank=40, vdim=24, scale=0.1, mlp=group_moe(8, 4, 1, 2, 16, 0.6))])


def aligned_gaparax():
    """Sizes near a real model's proportions, still small: several tiles of the tensor-core kernels."""
    return gaparax([sink_latent(heads=6, dim=128, rot=64, rank=160, vdim=96, scale=0.08, base=5e4, scaling=yarn(4.0, 256, 16.0, 1.0), mlp=relu2_dense(520)),
                    sigmoid_heads(heads=8, kv_heads=2, dim=128, vdim=104, chunk=200, scale=0.09, softcap=15.0, bias_max=90, mlp=group_moe(12, 4, 2, 4, 96)),
                    sigmoid_heads(heads=4, kv_heads=4, dim=64, vdim=64, chunk=131, scale=0.2, softcap=30.0, bias_max=200, mlp=group_moe(10, 5, 4, 6, 80, 2.5)),
                    sink_latent(heads=17, dim=48, rot=32, rank=96, vdim=40, scale=0.12, mlp=group_moe(8, 2, 1, 3, 64))], vocab=544, width=312, eps=1e-6, streams=2)
