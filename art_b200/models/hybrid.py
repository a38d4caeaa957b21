"""Hybrid decoders: models whose layers are listed one by one, each with its own sequence mixer and feed-forward.

A configuration consists of layers and of the frame around them.  A layer (``LayerSpec``) names

* a mixer: latent attention with a sliding window or a sink, grouped-query attention with a window or in chunks, HGRN2 or
  lightning linear attention, RWKV-style time mixing, a gated linear recurrent unit behind a short convolution, or several of
  these side by side on the same input, each with a factor (``parts``).  Grouped-query attention may rotate its queries and keys
  (either pairing, scaled frequencies), norm them (all heads together or each), squash its scores, weigh keys by sigmoids of
  scores with a bias by distance instead of a softmax, gate its heads or its result's columns and read another layer's keys and
  values;
* a feed-forward: PolyNorm, plain (``act(up)``), gated (``act(gate) * up``), a mixture of experts (gated or not, some of them the
  identity, chosen among all or among the best groups) with an optional shared expert, or none.

The frame (fields of ``HybridConfig``) is the design's: norms before, after, or before and after each sublayer, norm weights
stored as they are or around zero, a factor per column or a gate on each sublayer's result, a residual multiplier, a weighted
average over the results of all earlier layers, hyper-connections (several copies of the residual stream that every sublayer
reads and mixes), an embedding that is normalised, or scaled and given sinusoidal position vectors, an output table of its own
or the embedding's.

``HybridConfig`` answers the questions the engine asks of any configuration (``vocab_size``, ``hidden_size``,
``num_layers``, ``is_moe`` ...); ``from_design_dict`` reads a ``config.json`` whose ``architecture`` key names a design of
``ARCHITECTURES``.  ``tensor_shapes`` lists the checkpoint's tensors; ``check_weights`` compares a loaded checkpoint with
it.  The reference serves library models only (src/art/local/state.py); designs without a library are this package's own.
"""
from __future__ import annotations

import dataclasses
import math
from dataclasses import dataclass, field

import torch

SHIFT_MIXES = ("r", "k", "v", "g", "w")        # inputs of the token-shift mixer, in the order its kernels use
PART_NAMES = ("left", "right")                 # tensors of a parallel mixer's parts
RECURRENT = ("hgrn2", "wkv", "lightning", "rglru")
MAX_EXPERTS, MAX_TOP = 256, 16                 # what the router kernel holds
MAX_STREAMS = 8                                # ... and the one that mixes the copies of the residual stream
GATED_SUBLAYERS = ("latent_attention", "attention", "rglru", "parallel", "plain", "moe")      # whose input product takes a residual gate's rows, too


@dataclass
class LayerSpec:
    """One layer: mixer type, the mixer's sizes and constants, and its feed-forward."""
    type: str
    heads: int                                 # rglru: blocks of its gate matrices
    dim: int                                   # rglru: channels per block
    vdim: int
    ff: int = 0                                # width of a dense feed-forward, 0: none
    # attention
    rot_dim: int = 0                           # rotated dimensions of a head, 0: no rotation
    rot_pairs: str = "half"                    # a dimension's partner: half the rotated ones further ("half") or its neighbour ("next")
    rope_scaling: tuple[float, float, float, float] | None = None      # factor, original context, fast and slow turns (YaRN)
    kv_rank: int = 0
    kv_heads: int = 0
    scale: float = 1.0
    rope_base: float = 10000.0
    window: int = 0                            # keys seen, the token itself included; 0: all earlier ones
    chunk: int = 0                             # keys of the same chunk of the sequence only; 0: all earlier ones
    biases: bool = False                       # q, k and v projections have biases
    out_bias: bool = False                     # ... and the output projection
    qk_norm: bool = False                      # RMS norm over all heads of q together, and of k, before the rotation
    qk_norm_heads: bool = False                # ... over each head instead, with one head's weights
    head_temp: bool = False                    # scores have a learned factor per head (with qk_norm_heads)
    softcap: float = 0.0                       # scores pass softcap * tanh(score / softcap); 0: as they are
    sigmoid: bool = False                      # a key weighs sigmoid(score + its distance's bias + the head's), without normalisation
    bias_max: float = 0.0                      # distance at which the logarithmic buckets of the bias end
    bias_rows: int = 0                         # ... and their number (given by the tensor, not by the configuration)
    sink: bool = False                         # the softmax's denominator has a learned term per head (latent attention)
    head_gate: bool = False                    # heads are multiplied by the sigmoid of a projection of the input
    out_gate: bool = False                     # all columns of the heads are
    kv_from: int = -1                          # layer whose keys and values this one reads; -1: its own
    # wkv: width of the low-rank decay projection (given by its tensors, not by the configuration)
    decay_rank: int = 0
    decay: tuple[float, ...] = ()              # lightning: one factor per head
    conv: int = 1                              # rglru: taps of the short convolution
    parts: tuple["LayerSpec", ...] = ()        # parallel: mixers side by side, and the factor of each one's result
    part_scales: tuple[float, ...] = ()
    # feed-forward: "poly" (up, PolyNorm, down), "plain" (act(up), down), "gated" (act(gate) * up, down) or "moe" (experts)
    mlp: str = "poly"
    act: str = "silu"
    glu: bool = True                           # experts are act(gate) * up, down; else act(up), down
    experts: int = 0
    top: int = 0
    expert_ff: int = 0
    identity: int = 0                          # further outputs of the router that hand the input on
    router: str = "logits"                     # chooses by "logits" (+ bias, softmax over the chosen) or "scores" (softmax over all, + correction);
                                               # "softmax": by the softmax over all, which are the weights
    groups: int = 1                            # experts form equal groups of neighbours, of which the best ones can be chosen from
    group_keep: int = 1
    router_scale: float = 1.0                  # factor of the weights
    shared_ff: int = 0                         # shared expert, 0: none
    shared_gate: bool = False                  # the shared expert is multiplied by the sigmoid of a projection of the input

    @property
    def recurrent(self) -> bool:
        return self.type in RECURRENT or any(p.recurrent for p in self.parts)

    @property
    def has_mlp(self) -> bool:
        return self.ff > 0 or self.experts > 0

    def mixers(self) -> tuple["LayerSpec", ...]:
        """The single mixers of the layer."""
        return self.parts or (self,)


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
    # the frame
    pre_norms: bool = True                     # a norm before each sublayer; without, sublayers read the residual stream itself
    post_norms: bool = True                    # a norm behind each sublayer
    layer_scale: bool = False                  # each sublayer's result (behind its norm) has a factor per column
    residual_gate: bool = False                # each sublayer's result is multiplied by sigmoid(W h + b), h being its input
    streams: int = 0                           # hyper-connections: copies of the residual stream; 0: one stream, plain sums
    depth_average: bool = True                 # layer results are averaged with all earlier ones
    norm_offset: float = 0.0                   # added to the weights of the frame's norms
    embed_norm: bool = True
    embed_scale: float = 1.0
    position_base: float = 0.0                 # sinusoidal position vectors of this base are added to the embedding; 0: none
    tie_word_embeddings: bool = True

    is_moe = False                             # of the trainable families

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def recurrent(self) -> bool:
        """True when some layer carries a state from token to token (no prefix of a sequence can then be shared)."""
        return any(s.recurrent for s in self.layers)

    def kv_layer(self, i: int) -> int:
        """The layer whose keys and values layer ``i`` reads: its own, or the one it shares with."""
        return self.layers[i].kv_from if self.layers[i].kv_from >= 0 else i

    def norm_names(self, k: int) -> tuple[str | None, str | None]:
        """Tensors of sublayer ``k``'s (1: mixer, 2: feed-forward) norms before and behind it."""
        if not self.pre_norms:
            return None, f"norm{k}"
        return f"norm{k}", f"norm{k}b" if self.post_norms else None

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
        design = d["architecture"]
        if design not in ARCHITECTURES:
            raise ValueError(f"architecture {design!r} is not supported (supported: {', '.join(ARCHITECTURES)})")
        cfg = ARCHITECTURES[design](d, name)
        for i, s in enumerate(cfg.layers):
            _check_layer(i, s)
            if s.kv_from >= 0:
                _check_shared(cfg, i, s)
        _check_frame(cfg)
        return cfg


def _check_layer(i: int, s: LayerSpec) -> None:
    for p in s.mixers():
        if p.type == "attention" and (p.kv_heads <= 0 or p.heads % p.kv_heads):
            raise ValueError(f"layer {i}: {p.heads} query heads do not divide over {p.kv_heads} key heads")
        if p.type == "attention" and (p.rot_dim % 2 or p.rot_dim > p.dim):
            raise ValueError(f"layer {i}: rot.dims must be even and at most the head's {p.dim} dimensions, not {p.rot_dim}")
        if p.type == "lightning" and len(p.decay) != p.heads:
            raise ValueError(f"layer {i}: {len(p.decay)} decay factors for {p.heads} heads")
        if p.type in ("hgrn2", "wkv", "lightning") and max(p.dim, p.vdim) > 256:
            raise ValueError(f"layer {i}: {p.type} heads of more than 256 columns are not supported")
        if p.head_temp and not p.qk_norm_heads:
            raise ValueError(f"layer {i}: a factor per head goes with a norm of each head")
        if p.sigmoid and p.bias_max <= 0:
            raise ValueError(f"layer {i}: bias_max must be positive, not {p.bias_max}")
    if s.groups < 1 or (s.experts and ((s.experts + s.identity) % s.groups or not 1 <= s.group_keep <= s.groups)):
        raise ValueError(f"layer {i}: {s.group_keep} of {s.groups} groups of {s.experts + s.identity} experts are not supported")
    if s.experts and s.top > (s.experts + s.identity) // s.groups * s.group_keep:
        raise ValueError(f"layer {i}: {s.group_keep} groups have fewer than {s.top} experts")
    outputs = s.experts + s.identity
    if s.experts and not (0 < s.top <= min(outputs, MAX_TOP) and outputs <= MAX_EXPERTS):
        raise ValueError(f"layer {i}: {s.top} of {outputs} experts (at most {MAX_TOP} of {MAX_EXPERTS}) are not supported")


def _check_shared(cfg: HybridConfig, i: int, s: LayerSpec) -> None:
    src = cfg.layers[s.kv_from] if s.kv_from < i else None
    if src is None or src.type != "attention" or src.parts or src.kv_from >= 0:
        raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with keys and values of its own")
    if (src.kv_heads, src.dim, src.vdim) != (s.kv_heads, s.dim, s.vdim):
        raise ValueError(f"layer {i}: its key heads differ from those of layer {s.kv_from}, whose keys and values it reads")


def _check_frame(cfg: HybridConfig) -> None:
    if not 0 <= cfg.streams <= MAX_STREAMS:
        raise ValueError(f"{cfg.streams} streams are not supported (at most {MAX_STREAMS})")
    plain = cfg.pre_norms and not (cfg.post_norms or cfg.depth_average or cfg.embed_norm or cfg.layer_scale or cfg.position_base)
    if cfg.streams and not (plain and cfg.embed_scale == 1.0 and cfg.residual_mult == 1.0 and not any(s.type == "wkv" for s in cfg.layers)):
        raise ValueError("hyper-connections go with norms before the sublayers and nothing else around them")
    for i, s in enumerate(cfg.layers if cfg.residual_gate else ()):
        bad = [k for k in (s.type, s.mlp if s.has_mlp else "plain") if k not in GATED_SUBLAYERS]
        if bad or not cfg.pre_norms or cfg.post_norms:
            raise ValueError(f"layer {i}: a residual gate is not supported with {bad[0] if bad else 'these norms'}")


def distance_buckets(rows: int, reach: float, chunk: int = 0) -> list[int]:
    """Row of a distance bias's table for every distance from 0 on, up to the first one that has the row of all farther ones
    (or to the end of a chunk): a row per distance in the near half of the rows, then logarithmic up to ``reach``."""
    half = rows // 2
    if half < 1 or reach <= half:
        raise ValueError(f"a distance bias of {rows} rows up to distance {reach} is not supported")
    out: list[int] = []
    while not (out and (out[-1] == rows - 1 or len(out) in (chunk, 1 << 20))):
        n = len(out)
        out.append(n if n < half else min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half))))
    return out


def rope_frequencies(s: LayerSpec) -> tuple[list[float], float]:
    """One frequency per rotated pair and the factor of sine and cosine.  Scaled (YaRN; Peng et al., "YaRN: Efficient Context
    Window Extension of Large Language Models"): pairs that make few turns over the original context are slowed by the factor,
    those that make many are kept, with a linear ramp over the pairs in between."""
    n = s.rot_dim
    freq = [s.rope_base ** (-2.0 * j / n) for j in range(n // 2)]
    if s.rope_scaling is None:
        return freq, 1.0
    factor, original, fast, slow = s.rope_scaling

    def pair(turns: float) -> float:
        return n * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(s.rope_base))

    lo, hi = max(math.floor(pair(fast)), 0), min(math.ceil(pair(slow)), n - 1)
    for j in range(n // 2):
        ramp = min(1.0, max(0.0, (j - lo) / max(hi - lo, 0.001)))
        freq[j] = freq[j] / factor * ramp + freq[j] * (1.0 - ramp)
    return freq, 0.1 * math.log(factor) + 1.0


def _known(i: int, what: str, d: dict, keys: tuple[str, ...]) -> None:
    extra = sorted(k for k in set(d) - set(keys) if d[k] is not None)
    if extra:
        raise ValueError(f"layer {i}: {what} key{'s' if len(extra) > 1 else ''} {', '.join(map(repr, extra))} not supported")


def _mixer_kind(i: int, e: dict, supported: tuple[str, ...]) -> str:
    if e["type"] not in supported:
        raise ValueError(f"layer {i}: mixer {e['type']!r} is not supported (supported: {', '.join(supported)})")
    return e["type"]


def _mlp_kind(i: int, mlp: dict | None, supported: tuple[str, ...]) -> str | None:
    if mlp is None:
        return None
    kind = mlp.get("kind", "dense")
    if kind not in supported:
        raise ValueError(f"layer {i}: feed-forward kind {kind!r} is not supported (supported: {', '.join(supported)})")
    return kind


def _scaling(rot: dict) -> tuple[float, float, float, float] | None:
    return tuple(float(rot["scaling"][k]) for k in ("factor", "original", "fast", "slow")) if rot.get("scaling") else None


def _read_nikelix(d: dict, name: str) -> HybridConfig:
    layers = []
    for i, e in enumerate(d["layers"]):
        kind, m, mlp = _mixer_kind(i, e, ("latent_attention", "hgrn2", "wkv")), e["mixer"], e.get("mlp")
        _mlp_kind(i, mlp, ("dense",))
        spec = LayerSpec(kind, int(m["heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), int(mlp["ff"]) if mlp else 0)
        if kind == "latent_attention":
            rot = m["rot"]
            spec.rot_dim, spec.kv_rank, spec.rot_pairs = int(m["rot_dim"]), int(m["kv_rank"]), "next"
            spec.scale, spec.rope_base = float(m["scale"]), float(rot["base"])
            spec.window = int((m.get("mask") or {}).get("size", 0))
            if int(rot.get("dims", spec.rot_dim)) != spec.rot_dim:
                raise ValueError(f"layer {i}: rot.dims must equal rot_dim (the whole rotated part turns)")
            if spec.rot_dim % 2:
                raise ValueError(f"layer {i}: rot_dim must be even")
        layers.append(spec)
    return HybridConfig(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                        norm_eps=float(d["norm"]["eps"]), residual_mult=float(d["residual_mult"]), family="nikelix")


def _read_naselorn(d: dict, name: str) -> HybridConfig:
    layers = []
    for i, e in enumerate(d["layers"]):
        kind, m, mlp = _mixer_kind(i, e, ("parallel", "lightning")), e["mixer"], e.get("mlp")
        if kind == "lightning":
            spec = LayerSpec(kind, int(m["heads"]), int(m["dim"]), int(m["vdim"]), decay=tuple(float(x) for x in m["decay"]))
        else:
            a, r = m["left"], m["right"]
            width, blocks = int(r["width"]), int(r["blocks"])
            if width % blocks:
                raise ValueError(f"layer {i}: {width} channels do not divide over {blocks} blocks")
            parts = (LayerSpec("attention", int(a["heads"]), int(a["dim"]), int(a["vdim"]), kv_heads=int(a["kv_heads"]), scale=float(a["scale"]),
                               chunk=int((a.get("mask") or {}).get("size", 0)), biases=True, out_bias=True),
                     LayerSpec("rglru", blocks, width // blocks, width // blocks, conv=int(r["conv"])))
            spec = LayerSpec(kind, 0, 0, 0, parts=parts, part_scales=(float(m["left_scale"]), float(m["right_scale"])))
        ff = _mlp_kind(i, mlp, ("dense", "moe"))
        if ff == "dense":
            spec.mlp, spec.act, spec.ff = "gated", "relu", int(mlp["ff"])
        elif ff == "moe":
            spec.mlp, spec.expert_ff = "moe", int(mlp["expert"]["ff"])
            spec.experts, spec.top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
            spec.shared_ff = int(mlp["shared"]["ff"]) if mlp.get("shared") else 0
        layers.append(spec)
    return HybridConfig(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, norm_eps=float(d["norm"]["eps"]),
                        embed_scale=float(d["embedding"]["scale"]), **NASELORN_FRAME)


def _read_gaborax(d: dict, name: str) -> HybridConfig:
    layers = []
    for i, e in enumerate(d["layers"]):
        kind, m, mlp = _mixer_kind(i, e, ("attention", "attention_2")), e["mixer"], e.get("mlp")
        _known(i, "mixer", m, ("heads", "kv_heads", "dim", "vdim", "rot", "scale", "softcap", "kv_from"))
        first, rot = kind == "attention", m["rot"]
        _known(i, "rot", rot, ("base", "dims", "scaling"))
        spec = LayerSpec("attention", int(m["heads"]), int(m["dim"]), int(m["vdim"]), kv_heads=int(m["kv_heads"]), scale=float(m["scale"]),
                         rot_dim=int(rot["dims"]), rope_base=float(rot["base"]), rot_pairs="half" if first else "next", qk_norm=True,
                         biases=not first, head_gate=first, softcap=float(m.get("softcap") or 0.0))
        spec.rope_scaling = _scaling(rot)
        if m.get("kv_from") is not None:
            spec.kv_from = int(m["kv_from"])
            if spec.kv_from < 0:
                raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with keys and values of its own")
        if _mlp_kind(i, mlp, ("moe",)):
            r, shared = mlp["router"], mlp.get("shared")
            spec.mlp, spec.act, spec.glu, spec.router = "moe", "relu2", False, "scores"
            spec.expert_ff, spec.experts, spec.top, spec.identity = int(mlp["expert"]["ff"]), int(r["experts"]), int(r["top"]), int(r.get("identity") or 0)
            spec.shared_ff, spec.shared_gate = (int(shared["ff"]), True) if shared else (0, False)
        layers.append(spec)
    return HybridConfig(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, norm_eps=float(d["norm"]["eps"]),
                        **GABORAX_FRAME)


def _read_gaparax(d: dict, name: str) -> HybridConfig:
    layers = []
    for i, e in enumerate(d["layers"]):
        kind, m, mlp = _mixer_kind(i, e, ("attention", "latent_attention")), e["mixer"], e.get("mlp")
        spec = LayerSpec(kind, int(m["heads"]), int(m["dim"]), int(m["vdim"]), scale=float(m["scale"]))
        if kind == "attention":
            _known(i, "mixer", m, ("heads", "kv_heads", "dim", "vdim", "scale", "softcap", "bias_max", "mask"))
            _known(i, "mask", m.get("mask") or {}, ("size",))
            spec.kv_heads, spec.chunk = int(m["kv_heads"]), int((m.get("mask") or {}).get("size", 0))
            spec.softcap, spec.bias_max, spec.sigmoid = float(m.get("softcap") or 0.0), float(m["bias_max"]), True
            spec.qk_norm = spec.qk_norm_heads = spec.head_temp = spec.out_gate = True
        else:
            _known(i, "mixer", m, ("heads", "dim", "rot_dim", "kv_rank", "vdim", "rot", "scale"))
            rot = m["rot"]
            _known(i, "rot", rot, ("base", "dims", "scaling"))
            spec.rot_dim, spec.kv_rank, spec.rope_base, spec.rope_scaling = int(m["rot_dim"]), int(m["kv_rank"]), float(rot["base"]), _scaling(rot)
            spec.sink = True
            if int(rot.get("dims", spec.rot_dim)) != spec.rot_dim or spec.rot_dim % 2:
                raise ValueError(f"layer {i}: rot.dims must equal rot_dim, an even number (the whole rotated part turns)")
        ff = _mlp_kind(i, mlp, ("dense", "moe"))
        if ff == "dense":
            spec.mlp, spec.act, spec.ff = "plain", "relu2", int(mlp["ff"])
        elif ff == "moe":
            _known(i, "mlp", mlp, ("kind", "expert", "router"))
            r = mlp["router"]
            _known(i, "router", r, ("experts", "top", "groups", "scale"))
            spec.mlp, spec.router, spec.expert_ff, spec.experts, spec.top = "moe", "softmax", int(mlp["expert"]["ff"]), int(r["experts"]), int(r["top"])
            spec.router_scale = float(r.get("scale", 1.0))
            if r.get("groups"):
                spec.groups, spec.group_keep = int(r["groups"]["count"]), int(r["groups"]["keep"])
        layers.append(spec)
    return HybridConfig(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, norm_eps=float(d["norm"]["eps"]),
                        streams=int(d["streams"]), **GAPARAX_FRAME)


NASELORN_FRAME = dict(family="naselorn", post_norms=False, depth_average=False, norm_offset=1.0, embed_norm=False, position_base=10000.0,
                      tie_word_embeddings=False)
GABORAX_FRAME = dict(family="gaborax", pre_norms=False, post_norms=True, layer_scale=True, depth_average=False, norm_offset=1.0, embed_norm=False)
GAPARAX_FRAME = dict(family="gaparax", post_norms=False, depth_average=False, embed_norm=False, residual_gate=True, tie_word_embeddings=False)
ARCHITECTURES = {"Nikelix": _read_nikelix, "Naselorn": _read_naselorn, "Gaborax": _read_gaborax, "Gaparax": _read_gaparax}


def _mixer_shapes(s: LayerSpec, d: int) -> dict[str, tuple[int, ...]]:
    qk, v = s.heads * s.dim, s.heads * s.vdim
    if s.parts:
        return {f"{n}.{k}": t for n, p in zip(PART_NAMES, s.parts) for k, t in _mixer_shapes(p, d).items()}
    if s.type == "latent_attention":
        return {"q": (s.heads * (s.dim + s.rot_dim), d), "dkv": (s.kv_rank + s.rot_dim, d), "dkv.norm": (s.kv_rank,),
                "uk": (qk, s.kv_rank), "uv": (v, s.kv_rank), "o": (d, v), **({"sink": (s.heads,)} if s.sink else {})}
    if s.type == "hgrn2":
        return {"q": (qk, d), "f": (qk, d), "f.b": (qk,), "lower": (qk,), "v": (v, d), "norm": (s.vdim,), "o": (d, v)}
    if s.type == "lightning":
        return {"q": (qk, d), "k": (qk, d), "v": (v, d), "g": (v, d), "o": (d, v), "norm": (v,)}
    if s.type == "attention":
        own = {"q": (qk, d)}
        if s.kv_from < 0:
            own.update({"k": (s.kv_heads * s.dim, d), "v": (s.kv_heads * s.vdim, d)})
        out = {**own, "o": (d, v)}
        if s.biases:
            out.update({k + ".b": (t[0],) for k, t in own.items()})
        if s.out_bias:
            out["o.b"] = (d,)
        if s.qk_norm:
            out.update({k + ".norm": (s.dim if s.qk_norm_heads else own[k][0],) for k in "qk" if k in own})
        if s.head_gate or s.out_gate:
            out["g"] = (v if s.out_gate else s.heads, d)
        if s.head_temp:
            out["temp"] = (s.heads,)
        if s.sigmoid:
            out.update({"rel": (s.bias_rows, s.heads), "pb": (s.heads,)})
        return out
    if s.type == "rglru":
        gates = {k: t for g in ("ra", "ri") for k, t in ((g, (s.heads, s.dim, s.dim)), (g + ".b", (s.heads, s.dim)))}
        return {"y": (qk, d), "y.b": (qk,), "x": (qk, d), "x.b": (qk,), "conv": (qk, s.conv), "conv.b": (qk,), **gates, "lam": (qk,), "o": (d, qk)}
    out = {"mu." + m: (d,) for m in SHIFT_MIXES}
    out.update({m: (qk, d) for m in "rkvg"})
    out.update({"w1": (s.decay_rank, d), "w2": (qk, s.decay_rank), "w0": (qk,), "u": (s.heads, s.dim), "norm": (qk,), "o": (d, qk)})
    return out


def _mlp_shapes(s: LayerSpec, d: int) -> dict[str, tuple[int, ...]]:
    def glu(pre: str, ff: int) -> dict[str, tuple[int, ...]]:
        return {pre + "gate": (ff, d), pre + "up": (ff, d), pre + "down": (d, ff)}

    if s.mlp == "poly":
        return {"up": (s.ff, d), "down": (d, s.ff), "act": (4,)}
    if s.mlp == "plain":
        return {"up": (s.ff, d), "down": (d, s.ff)}
    if s.mlp == "gated":
        return glu("", s.ff)
    form = glu if s.glu else lambda pre, ff: {pre + "up": (ff, d), pre + "down": (d, ff)}
    out = {k: t for e in range(s.experts) for k, t in form(f"e{e}.", s.expert_ff).items()}
    n = s.experts + s.identity
    out["router"] = (n, d)
    if s.router != "softmax":
        out["router.b" if s.router == "logits" else "correction"] = (n,)
    if s.shared_ff:
        out.update(form("shared.", s.shared_ff))
        if s.shared_gate:
            out["shared.sg"] = (1, d)
    return out


def tensor_shapes(cfg: HybridConfig) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor of a checkpoint.  The decay rank of a wkv layer and the rows of a distance bias are taken
    from the layer's spec."""
    d = cfg.hidden_size
    out: dict[str, tuple[int, ...]] = {"embed": (cfg.vocab_size, d), "final.norm": (d,)}
    if cfg.embed_norm:
        out["embed.norm"] = (d,)
    if not cfg.tie_word_embeddings:
        out["head"] = (cfg.vocab_size, d)
    for i, s in enumerate(cfg.layers):
        p = f"l{i}."
        for k in (1, 2) if s.has_mlp else (1,):
            out.update({p + n: (d,) for n in cfg.norm_names(k) if n})
            if cfg.layer_scale:
                out[f"{p}ls{k}"] = (d,)
            if cfg.residual_gate:
                out.update({f"{p}rg{k}": (d, d), f"{p}rg{k}.b": (d,)})
            if cfg.streams:
                n = cfg.streams
                out.update({f"{p}hc{k}.in": (n,), f"{p}hc{k}.out": (n,), f"{p}hc{k}.mix": (n, n)})
        if s.has_mlp:
            out.update({p + "mlp." + k: t for k, t in _mlp_shapes(s, d).items()})
        out.update({p + "mix." + k: t for k, t in _mixer_shapes(s, d).items()})
        if cfg.depth_average:
            out[p + "dwa"] = (i + 2,)
    return out


def check_weights(cfg: HybridConfig, w: dict[str, torch.Tensor]) -> None:
    """Fills in the sizes that only the tensors give and raises when a tensor is missing or has another shape."""
    for i, s in enumerate(cfg.layers):
        w1 = w.get(f"l{i}.mix.w1")
        if s.type == "wkv" and w1 is not None:
            s.decay_rank = int(w1.shape[0])
        for p, pre in zip(s.mixers(), PART_NAMES if s.parts else ("",)):
            rel = w.get(f"l{i}.mix.{pre + '.' if pre else ''}rel")
            if p.sigmoid and rel is not None:
                p.bias_rows = int(rel.shape[0])
                distance_buckets(p.bias_rows, p.bias_max)
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
        for p in s.mixers():
            if p.sigmoid and not p.bias_rows:
                p.bias_rows = max(2, min(32, int(p.bias_max) // 2 * 2))
    w: dict[str, torch.Tensor] = {}
    frame = ("norm1", "norm1b", "norm2", "norm2b", "final.norm", "embed.norm")
    for k, shape in tensor_shapes(cfg).items():
        leaf = k.split(".", 2)[-1] if k.startswith("l") else k
        if "norm" in leaf:
            w[k] = rnd(*shape, std=0.1, mean=1.0 - (cfg.norm_offset if leaf in frame or k.split(".")[-1] in frame else 0.0))
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
        elif leaf.endswith("lam"):             # memories from a token to some thousand tokens
            w[k] = uni(*shape, lo=-8.0, hi=1.0)
        elif leaf in ("ls1", "ls2"):
            w[k] = rnd(*shape, std=0.2, mean=0.8)
        elif leaf == "correction":             # moves a choice now and then
            w[k] = rnd(*shape, std=0.3 / shape[0])
        elif leaf in ("in", "out") and ".hc" in k:      # streams stay of one size: about their mean goes in, a share comes out
            w[k] = rnd(*shape, std=0.3 / shape[0], mean=1.0 / shape[0] if leaf == "in" else 0.8)
        elif leaf == "mix":
            w[k] = (torch.eye(shape[0], device=device) * 0.8 + 0.2 / shape[0]).to(dtype) + rnd(*shape, std=0.05)
        elif leaf == "temp":
            w[k] = rnd(*shape, std=0.2, mean=1.0)
        elif leaf in ("rel", "pb", "sink"):
            w[k] = rnd(*shape, std=0.7)
        elif leaf in ("u", "f.b", "b") or leaf.endswith(".b"):
            w[k] = rnd(*shape, std=0.5)
        else:
            w[k] = rnd(*shape, std=shape[-1] ** -0.5)
    return w


def _preset(name: str, width: int, ff: int, heads: int, n_layers: int, vocab: int = 32000, window: int = 1024) -> HybridConfig:
    """``n_layers`` layers that repeat (latent attention, hgrn2, wkv, hgrn2) at the proportions of a model this wide."""
    hd = width // heads
    la = LayerSpec("latent_attention", heads, 128, 128, ff, rot_dim=64, kv_rank=512, scale=192 ** -0.5, rope_base=5e5, rot_pairs="next", window=window)
    hg = LayerSpec("hgrn2", heads, hd, hd, ff)
    wk = LayerSpec("wkv", width // 64, 64, 64, ff, decay_rank=64)
    cycle = (la, hg, wk, hg)
    return HybridConfig(name=name, vocab_size=vocab, hidden_size=width,
                        layers=[dataclasses.replace(cycle[i % 4]) for i in range(n_layers)], residual_mult=0.5)


def _naselorn_preset(name: str, width: int, n_layers: int, experts: int, top: int, expert_ff: int, shared_ff: int, dense_ff: int,
                     vocab: int = 32000, chunk: int = 1024) -> HybridConfig:
    """``n_layers`` layers, every fourth one parallel, the others lightning; the first has a dense feed-forward."""
    hd = 128
    decay = tuple(1 - 2.0 ** (-1 - 7.0 * h / max(1, width // hd - 1)) for h in range(width // hd))
    li = LayerSpec("lightning", width // hd, hd, hd, decay=decay)
    parts = (LayerSpec("attention", width // hd, hd, hd, kv_heads=max(1, width // hd // 4), scale=hd ** -0.5, chunk=chunk, biases=True, out_bias=True),
             LayerSpec("rglru", width // 256, 256, 256, conv=4))
    pa = LayerSpec("parallel", 0, 0, 0, parts=parts, part_scales=(0.5, 0.5))
    layers = [dataclasses.replace(pa if i % 4 == 3 else li, mlp="moe", experts=experts, top=top, expert_ff=expert_ff, shared_ff=shared_ff)
              for i in range(n_layers)]
    layers[0] = dataclasses.replace(li, mlp="gated", act="relu", ff=dense_ff)
    return HybridConfig(name=name, vocab_size=vocab, hidden_size=width, layers=layers, embed_scale=width ** 0.5, **NASELORN_FRAME)


def _gaborax_preset(name: str, width: int, n_layers: int, experts: int, identity: int, top: int, expert_ff: int, shared_ff: int,
                    vocab: int = 32000) -> HybridConfig:
    """``n_layers`` layers that alternate between the two kinds of attention; every fourth one reads the keys and values of the
    layer two before it."""
    hd, heads = 128, width // 128
    one = LayerSpec("attention", heads, hd, hd, kv_heads=max(1, heads // 4), scale=hd ** -0.5, rot_dim=hd, rope_base=5e5, qk_norm=True, mlp="moe",
                    act="relu2", glu=False, router="scores", experts=experts, identity=identity, top=top, expert_ff=expert_ff, shared_ff=shared_ff,
                    shared_gate=True)
    a, b = dataclasses.replace(one, head_gate=True), dataclasses.replace(one, rot_pairs="next", biases=True, softcap=50.0, rope_scaling=(4.0, 8192, 32, 1))
    layers = [dataclasses.replace(b if i % 2 else a, kv_from=i - 2 if i % 4 == 2 else -1) for i in range(n_layers)]
    return HybridConfig(name=name, vocab_size=vocab, hidden_size=width, layers=layers, **GABORAX_FRAME)


def _gaborax_tiny() -> HybridConfig:
    moe = dict(mlp="moe", act="relu2", glu=False, router="scores", experts=6, identity=3, top=2, expert_ff=48, shared_ff=80, shared_gate=True)
    a = LayerSpec("attention", 4, 32, 24, kv_heads=2, scale=0.2, rot_dim=16, qk_norm=True, head_gate=True, **moe)
    b = LayerSpec("attention", 6, 24, 40, kv_heads=3, scale=0.25, rot_dim=24, rot_pairs="next", rope_scaling=(2.0, 256, 16, 1), qk_norm=True, biases=True,
                  softcap=20.0, **moe)
    return HybridConfig("gaborax-tiny", 512, 128, [a, b, dataclasses.replace(a, kv_from=0)], **GABORAX_FRAME)


def _gaparax_preset(name: str, width: int, n_layers: int, experts: int, top: int, expert_ff: int, dense_ff: int, vocab: int = 32000,
                    chunk: int = 1024) -> HybridConfig:
    """``n_layers`` layers, every fourth one latent attention, the others chunked attention; the first has a dense feed-forward."""
    hd, heads = 128, width // 128
    la = LayerSpec("latent_attention", heads, 128, 128, rot_dim=64, kv_rank=512, scale=192 ** -0.5, rope_base=5e5, rope_scaling=(4.0, 8192, 32, 1), sink=True)
    at = LayerSpec("attention", heads, hd, hd, kv_heads=max(1, heads // 4), scale=hd ** -0.5, chunk=chunk, qk_norm=True, qk_norm_heads=True, head_temp=True,
                   softcap=30.0, sigmoid=True, bias_max=256, out_gate=True)
    moe = dict(mlp="moe", router="softmax", experts=experts, top=top, groups=8, group_keep=4, router_scale=2.5, expert_ff=expert_ff)
    layers = [dataclasses.replace(la if i % 4 == 3 else at, **moe) for i in range(n_layers)]
    layers[0] = dataclasses.replace(at, mlp="plain", act="relu2", ff=dense_ff)
    return HybridConfig(name=name, vocab_size=vocab, hidden_size=width, layers=layers, streams=2, **GAPARAX_FRAME)


def _gaparax_tiny() -> HybridConfig:
    moe = dict(mlp="moe", router="softmax", experts=6, top=3, groups=3, group_keep=2, router_scale=1.5, expert_ff=48)
    at = LayerSpec("attention", 4, 32, 24, kv_heads=2, scale=0.2, chunk=40, qk_norm=True, qk_norm_heads=True, head_temp=True, softcap=15.0, sigmoid=True,
                   bias_max=60, out_gate=True)
    la = LayerSpec("latent_attention", 3, 24, 40, rot_dim=16, kv_rank=56, scale=0.15, rope_scaling=(3.0, 128, 16, 1), sink=True)
    return HybridConfig("gaparax-tiny", 512, 128, [dataclasses.replace(at, mlp="plain", act="relu2", ff=200), dataclasses.replace(la, **moe), at], streams=3,
                        **GAPARAX_FRAME)


HYBRID_PRESETS: dict[str, HybridConfig] = {
    "nikelix-tiny": HybridConfig("nikelix-tiny", 512, 128, [
        LayerSpec("hgrn2", 2, 24, 40, 192), LayerSpec("latent_attention", 3, 16, 24, 256, rot_dim=8, kv_rank=48, scale=0.2,
                                                       rope_base=1e4, rot_pairs="next", window=24),
        LayerSpec("wkv", 4, 16, 16, 0, decay_rank=8)], residual_mult=0.7),
    "nikelix-1b": _preset("nikelix-1b", 2048, 8192, 16, 16),
    "nikelix-7b": _preset("nikelix-7b", 4096, 16384, 32, 32),
    "naselorn-tiny": HybridConfig("naselorn-tiny", 512, 128, [
        LayerSpec("lightning", 2, 24, 40, 176, decay=(0.7, 0.97), mlp="gated", act="relu"),
        LayerSpec("parallel", 0, 0, 0, mlp="moe", experts=6, top=2, expert_ff=48, shared_ff=80, part_scales=(0.7, 0.4), parts=(
            LayerSpec("attention", 4, 16, 24, kv_heads=2, scale=0.25, chunk=20, biases=True, out_bias=True), LayerSpec("rglru", 3, 20, 20, conv=3)))],
        embed_scale=8.0, **NASELORN_FRAME),
    "naselorn-2b-a1b": _naselorn_preset("naselorn-2b-a1b", 2048, 16, 64, 8, 512, 1024, 6144),
    "naselorn-14b-a4b": _naselorn_preset("naselorn-14b-a4b", 4096, 16, 64, 8, 1024, 2048, 12288),
    "gaborax-tiny": _gaborax_tiny(),
    "gaborax-2b-a1b": _gaborax_preset("gaborax-2b-a1b", 2048, 16, 64, 8, 8, 768, 1536),
    "gaborax-14b-a4b": _gaborax_preset("gaborax-14b-a4b", 4096, 16, 64, 8, 8, 1536, 3072),
    "gaparax-tiny": _gaparax_tiny(),
    "gaparax-2b-a1b": _gaparax_preset("gaparax-2b-a1b", 2048, 16, 64, 8, 512, 8192),
    "gaparax-14b-a4b": _gaparax_preset("gaparax-14b-a4b", 4096, 16, 64, 8, 1024, 16384),
}
