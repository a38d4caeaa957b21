"""Hybrid decoders: models whose layers are listed one by one, each with its own sequence mixer.

A hybrid configuration names, per layer, a mixer (latent attention with a sliding window, HGRN2 linear attention,
RWKV-style time mixing) with its sizes, and a feed-forward (dense PolyNorm, or none).  The frame around the sublayers is
fixed by the design: RMS norms before and after each sublayer, a residual multiplier, a weighted average over the results
of all earlier layers, a normalised embedding, tied output.

``HybridConfig`` answers the questions the engine asks of any configuration (``vocab_size``, ``hidden_size``,
``num_layers``, ``is_moe`` ...); ``from_design_dict`` reads a ``config.json`` whose ``architecture`` key names a design of
``ARCHITECTURES``.  ``tensor_shapes`` lists the checkpoint's tensors; ``check_weights`` compares a loaded checkpoint with
it.  The reference serves library models only (src/art/local/state.py); designs without a library are this package's own.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

MIXERS = ("latent_attention", "hgrn2", "wkv")
SHIFT_MIXES = ("r", "k", "v", "g", "w")        # inputs of the token-shift mixer, in the order its kernels use


@dataclass
class LayerSpec:
    """One layer: mixer type, the mixer's sizes and constants, width of the feed-forward (0: none)."""
    type: str
    heads: int
    dim: int
    vdim: int
    ff: int = 0
    # latent attention
    rot_dim: int = 0
    kv_rank: int = 0
    scale: float = 1.0
    rope_base: float = 10000.0
    window: int = 0                            # keys seen, the token itself included; 0: all earlier ones
    # wkv: width of the low-rank decay projection (given by its tensors, not by the configuration)
    decay_rank: int = 0

    @property
    def recurrent(self) -> bool:
        return self.type != "latent_attention"


@dataclass
class HybridConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: list[LayerSpec] = field(default_factory=list)
    norm_eps: float = 1e-5
    residual_mult: float = 1.0
    family: str = "nikelix"
    max_position_embeddings: int = 1 << 20

    is_moe = False
    tie_word_embeddings = True

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def recurrent(self) -> bool:
        """True when some layer carries a state from token to token (no prefix of a sequence can then be shared)."""
        return any(s.recurrent for s in self.layers)

    def num_params(self) -> int:
        n = 0
        for shape in tensor_shapes(self).values():
            k = 1
            for s in shape:
                k *= s
            n += k
        return n

    @classmethod
    def from_design_dict(cls, d: dict, name: str = "hybrid") -> "HybridConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            kind, m, mlp = e["type"], e["mixer"], e.get("mlp")
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: mixer {kind!r} is not supported (supported: {', '.join(MIXERS)})")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not supported (supported: dense)")
            spec = LayerSpec(kind, int(m["heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), int(mlp["ff"]) if mlp else 0)
            if kind == "latent_attention":
                rot = m["rot"]
                spec.rot_dim, spec.kv_rank = int(m["rot_dim"]), int(m["kv_rank"])
                spec.scale, spec.rope_base = float(m["scale"]), float(rot["base"])
                spec.window = int((m.get("mask") or {}).get("size", 0))
                if int(rot.get("dims", spec.rot_dim)) != spec.rot_dim:
                    raise ValueError(f"layer {i}: rot.dims must equal rot_dim (the whole rotated part turns)")
                if spec.rot_dim % 2:
                    raise ValueError(f"layer {i}: rot_dim must be even")
            layers.append(spec)
        return cls(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                   norm_eps=float(d["norm"]["eps"]), residual_mult=float(d["residual_mult"]),
                   family=str(d["architecture"]).lower())


ARCHITECTURES = {"Nikelix": HybridConfig.from_design_dict}


def tensor_shapes(cfg: HybridConfig) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor of a checkpoint.  The decay rank of a wkv layer is taken from its spec."""
    d = cfg.hidden_size
    out: dict[str, tuple[int, ...]] = {"embed": (cfg.vocab_size, d), "embed.norm": (d,), "final.norm": (d,)}
    for i, s in enumerate(cfg.layers):
        p = f"l{i}."
        out[p + "norm1"] = out[p + "norm1b"] = (d,)
        x = p + "mix."
        qk, v = s.heads * s.dim, s.heads * s.vdim
        if s.type == "latent_attention":
            out[x + "q"] = (s.heads * (s.dim + s.rot_dim), d)
            out[x + "dkv"] = (s.kv_rank + s.rot_dim, d)
            out[x + "dkv.norm"] = (s.kv_rank,)
            out[x + "uk"], out[x + "uv"] = (qk, s.kv_rank), (v, s.kv_rank)
            out[x + "o"] = (d, v)
        elif s.type == "hgrn2":
            out[x + "q"] = out[x + "f"] = (qk, d)
            out[x + "f.b"] = out[x + "lower"] = (qk,)
            out[x + "v"], out[x + "norm"], out[x + "o"] = (v, d), (s.vdim,), (d, v)
        else:
            for m in SHIFT_MIXES:
                out[x + "mu." + m] = (d,)
            for m in "rkvg":
                out[x + m] = (qk, d)
            out[x + "w1"], out[x + "w2"], out[x + "w0"] = (s.decay_rank, d), (qk, s.decay_rank), (qk,)
            out[x + "u"], out[x + "norm"], out[x + "o"] = (s.heads, s.dim), (qk,), (d, qk)
        if s.ff:
            out[p + "norm2"] = out[p + "norm2b"] = (d,)
            out[p + "mlp.up"], out[p + "mlp.down"], out[p + "mlp.act"] = (s.ff, d), (d, s.ff), (4,)
        out[p + "dwa"] = (i + 2,)
    return out


def check_weights(cfg: HybridConfig, w: dict[str, torch.Tensor]) -> None:
    """Fills in the decay ranks from the tensors and raises when a tensor is missing or has another shape."""
    for i, s in enumerate(cfg.layers):
        w1 = w.get(f"l{i}.mix.w1")
        if s.type == "wkv" and w1 is not None:
            s.decay_rank = int(w1.shape[0])
    for k, shape in tensor_shapes(cfg).items():
        if k not in w:
            raise ValueError(f"checkpoint of {cfg.name} lacks tensor {k!r}")
        if tuple(w[k].shape) != shape:
            raise ValueError(f"tensor {k!r}: shape {tuple(w[k].shape)} in the checkpoint, {shape} by the configuration")


def init_hybrid_weights(cfg: HybridConfig, seed: int = 0, dtype: torch.dtype = torch.float32,
                        device: str | torch.device = "cpu") -> dict[str, torch.Tensor]:
    """Random weights whose activations keep a useful range: fan-in scaled matrices, norm weights around 1, decays and
    lower bounds spread over short and long memories."""
    g = torch.Generator(device=device).manual_seed(seed)

    def rnd(*shape: int, std: float = 1.0, mean: float = 0.0) -> torch.Tensor:
        return (torch.randn(*shape, generator=g, device=device, dtype=torch.float32) * std + mean).to(dtype)

    def uni(*shape: int, lo: float = 0.0, hi: float = 1.0) -> torch.Tensor:
        return (torch.rand(*shape, generator=g, device=device, dtype=torch.float32) * (hi - lo) + lo).to(dtype)

    for s in cfg.layers:
        if s.type == "wkv" and not s.decay_rank:
            s.decay_rank = max(8, cfg.hidden_size // 64 // 8 * 8)
    w: dict[str, torch.Tensor] = {}
    for k, shape in tensor_shapes(cfg).items():
        leaf = k.split(".", 2)[-1] if k.startswith("l") else k
        if "norm" in leaf:
            w[k] = rnd(*shape, std=0.1, mean=1.0)
        elif k.endswith(".dwa"):
            t = torch.full(shape, 0.3 / max(1, shape[0] - 1), device=device)
            t[-1] = 0.8
            w[k] = t.to(dtype)
        elif leaf == "act":
            w[k] = torch.tensor([0.8, 0.3, 0.2, 0.05], device=device).to(dtype)
        elif leaf == "lower":
            w[k] = uni(*shape, hi=0.95)
        elif leaf == "w0":
            w[k] = uni(*shape, lo=-6.0, hi=0.0)
        elif leaf.startswith("mu."):
            w[k] = uni(*shape)
        elif leaf in ("u", "f.b"):
            w[k] = rnd(*shape, std=0.5)
        else:
            w[k] = rnd(*shape, std=shape[-1] ** -0.5)
    return w


def _preset(name: str, width: int, ff: int, heads: int, n_layers: int, vocab: int = 32000, window: int = 1024) -> HybridConfig:
    """``n_layers`` layers that repeat (latent attention, hgrn2, wkv, hgrn2) at the proportions of a model this wide."""
    hd = width // heads
    la = LayerSpec("latent_attention", heads, 128, 128, ff, rot_dim=64, kv_rank=512, scale=192 ** -0.5, rope_base=5e5, window=window)
    hg = LayerSpec("hgrn2", heads, hd, hd, ff)
    wk = LayerSpec("wkv", width // 64, 64, 64, ff, decay_rank=64)
    import dataclasses

    cycle = (la, hg, wk, hg)
    return HybridConfig(name=name, vocab_size=vocab, hidden_size=width,
                        layers=[dataclasses.replace(cycle[i % 4]) for i in range(n_layers)], residual_mult=0.5)


HYBRID_PRESETS: dict[str, HybridConfig] = {
    "nikelix-tiny": HybridConfig("nikelix-tiny", 512, 128, [
        LayerSpec("hgrn2", 2, 24, 40, 192), LayerSpec("latent_attention", 3, 16, 24, 256, rot_dim=8, kv_rank=48, scale=0.2,
                                                       rope_base=1e4, window=24),
        LayerSpec("wkv", 4, 16, 16, 0, decay_rank=8)], residual_mult=0.7),
    "nikelix-1b": _preset("nikelix-1b", 2048, 8192, 16, 16),
    "nikelix-7b": _preset("nikelix-7b", 4096, 16384, 32, 32),
}
