"""Execution of hybrid decoders (``models/hybrid.py``) for the rollout engine.

One batch is ragged: every sequence brings its next tokens, whether one decoded token or a portion of its prompt, and all
of them go through the layers together.  ``Ragged`` describes it to the kernels: rows of the sequences one after another
(``cu_q``), positions, cache rows, block tables, state slots.  Sequences with few new tokens come first, so that a row
range tells which form of attention a row takes: short ones read the cache where it lies (latent attention: the absorbed
form), longer portions gather what they see and run on prompt kernels (latent attention: expanded keys and values).

A batch of single tokens (decoding) leaves its projections as split-K partial sums in fp32 workspaces, which the kernel
that follows finishes and clears, as the engine's other models do.

Every sublayer is ``(norm ->) mixer or feed-forward -> (norm ->) residual``; the step from one to the next (a mixture's weighted
sum, bias, gate, post-norm and factors, residual multiplier, depth average or mixing of hyper-connected streams, next input norm:
what the design has of them) is one kernel over the fp32 residual stream (``ops.hybrid.residual_step``).  A gate on a sublayer's
result is further rows of the sublayer's input product.  Mixers side by side share one input and one output product: their
factors scale what enters the latter.
Operands of the matrix products are bf16; with ``dtype=torch.float32`` everything is fp32, products included, through the
same layer code.

Decoding several tokens per call, CUDA graphs, sampling and logit processing come from
:class:`~art_b200.engine.runner.DeviceRunner`.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..models.hybrid import PART_NAMES, SHIFT_MIXES, HybridConfig, LayerSpec, check_weights, distance_buckets, rope_frequencies
from ..ops import hybrid as hy
from ..ops.hybrid import Out, Sublayer, as_out, pad
from .runner import DeviceRunner, SeqView


@dataclass
class Ragged:
    """A batch on the device.  ``single``: every sequence brings exactly one token (row m = sequence m)."""
    M: int
    n_seqs: int
    tokens: torch.Tensor        # int64 [M]
    pos: torch.Tensor           # int32 [M]
    slot: torch.Tensor          # int32 [M]   cache row of the token, -1: not written
    row_seq: torch.Tensor       # int32 [M]
    cu_q: torch.Tensor          # int32 [n_seqs + 1]
    ctx: torch.Tensor           # int32 [n_seqs]  tokens after this step; 0: padding
    state_slot: torch.Tensor    # int32 [n_seqs]
    bt: torch.Tensor            # int32 [n_seqs, max_blocks]
    single: bool
    # portions that attend in the expanded form, in row order behind n_abs shorter rows: (sequence, tokens before, tokens)
    portions: list[tuple[int, int, int]] = field(default_factory=list)
    n_abs: int = 0
    reach: int = 0              # upper bound of the tokens a short row may attend to
    plans: dict = field(default_factory=dict)
    kept: dict = field(default_factory=dict)      # gathered keys and values that a later layer reads, too

    def plan(self, window: int, chunk: int = 0) -> hy.PrefillPlan:
        p = self.plans.get((window, chunk))
        if p is None:
            p = self.plans[window, chunk] = hy.plan_prefill(self.portions, window, self.tokens.device, chunk)
        return p


# Portions up to this many tokens read the cache row by row: gathering (and, of latents, expanding) a window's keys and values
# for them would cost more.
ABSORB_MAX = 16
# Sizes the tensor-core kernels hold in shared memory and registers; beyond them the scalar absorbed form serves.
LATENT_TC_MAX = 768         # cached row: latent + rotated part
PREFILL_VALUE_MAX, PREFILL_KEY_MAX = 128, 320


# Kernel sources of each mechanism (what a fresh checkout has to compile before it can run a model's layers)
_GEMM = {"gemm_tcgen05", "gemm_tcgen05_2cta", "gemm_splitk", "gemm_f32"}
_SCAN = {"linear_scan"}
KERNEL_SOURCES = {
    "latent_attention": {"latent_attn", "latent_decode", "latent_prefill", "latent_prefill_tc", "gemm_batched"},
    "attention": {"gqa_attn", "latent_prefill", "latent_prefill_tc"}, "hgrn2": _SCAN, "wkv": _SCAN | {"gemm_batched"},
    "lightning": _SCAN | {"lightning_prefill"}, "rglru": {"rglru", "gemm_batched"}, "moe": {"moe", "gemm_grouped", "lora_wgrad"}}


def kernel_sources(cfg: HybridConfig) -> set[str]:
    """The kernel sources that the layers of a model run on."""
    kinds = {m.type for s in cfg.layers for m in s.mixers()} | {s.mlp for s in cfg.layers if s.has_mlp}
    return _GEMM | {"hybrid_rows"} | {f for k in kinds for f in KERNEL_SOURCES.get(k, ())}


class HybridRunner(DeviceRunner):
    mixed_steps = True
    # One-CTA and CTA-pair products follow one another directly here (per-head products in front of an output projection);
    # with overlapping launches their tensor-memory allocations would meet on an SM.  Full stream order between kernels.
    overlap_launches = False

    def __init__(self, cfg: HybridConfig, kv, base: dict[str, torch.Tensor], *, device="cuda", dtype: torch.dtype = torch.bfloat16,
                 max_loras: int = 0):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"hybrid models run in bfloat16 or float32, not {dtype}")
        check_weights(cfg, base)
        self.cfg, self.kv, self.device, self.dtype = cfg, kv, torch.device(device), dtype
        self.exact32 = dtype == torch.float32
        self.max_loras = max_loras
        self.dp = pad(cfg.hidden_size)
        wide = any(m.type in ("latent_attention", "attention") and
                   (m.vdim > PREFILL_VALUE_MAX or pad(m.dim, 16) + pad(m.rot_dim, 16) > PREFILL_KEY_MAX) for s in cfg.layers for m in s.mixers())
        self.shared_kv = {s.kv_from for s in cfg.layers if s.kv_from >= 0}
        self.absorb_max = 1 << 30 if self.exact32 or wide else ABSORB_MAX
        self._load(base)
        self._buf: dict = {}

    # -- weights ------------------------------------------------------------------------------------
    def _mat(self, w: torch.Tensor, rows: int | None = None, cols: int | None = None) -> torch.Tensor:
        """A matrix as GEMM operand: operand dtype, rows and columns padded with zeros (default: to multiples of 8)."""
        out = torch.zeros(rows or pad(w.shape[0]), cols or pad(w.shape[1]), dtype=self.dtype, device=self.device)
        out[:w.shape[0], :w.shape[1]] = w.to(self.device)
        return out

    def _vec(self, w: torch.Tensor, n: int | None = None) -> torch.Tensor:
        w = w.reshape(-1).to(self.device, torch.float32)
        out = torch.zeros(n or w.numel(), dtype=torch.float32, device=self.device)
        out[:w.numel()] = w
        return out

    def _heads_in(self, w: torch.Tensor, heads: int, vdim: int) -> torch.Tensor:
        """An output projection whose input keeps every head's ``vdim`` values at a pitch of ``pad(vdim)``."""
        d, vp = w.shape[0], pad(vdim)
        out = torch.zeros(self.dp, heads, vp, dtype=self.dtype, device=self.device)
        out[:d, :, :vdim] = w.to(self.device).view(d, heads, vdim)
        return out.view(self.dp, heads * vp)

    def _glu(self, gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
        """gate | up as one operand, rows interleaved in blocks of 16; the width is padded to a multiple of 16."""
        ff = pad(gate.shape[0], 16)
        g, u = self._mat(gate, ff, self.dp), self._mat(up, ff, self.dp)
        return torch.stack([g.view(-1, 16, self.dp), u.view(-1, 16, self.dp)], 1).reshape(2 * ff, self.dp)

    def _load(self, base: dict[str, torch.Tensor]) -> None:
        cfg, dp = self.cfg, self.dp
        V, d = cfg.vocab_size, cfg.hidden_size
        table = self._mat(base["embed"], pad(V), dp)
        self._head = table if cfg.tie_word_embeddings else self._mat(base["head"], pad(V), dp)
        self.embed, self.lm_head = table[:V], self._head[:V]

        def norm(w: torch.Tensor) -> torch.Tensor:
            out = self._vec(w, dp)
            out[:d] += cfg.norm_offset
            return out

        self.embed_norm = norm(base["embed.norm"]) if cfg.embed_norm else None
        self.final_norm = norm(base["final.norm"])
        self.pos_freq = None
        if cfg.position_base > 0:
            self.pos_freq = torch.tensor([cfg.position_base ** (-2.0 * i / d) for i in range(dp // 2)], dtype=torch.float64).to(self.device)
        self.layers = []
        for i, s in enumerate(cfg.layers):
            w = {k[len(f"l{i}."):]: t for k, t in base.items() if k.startswith(f"l{i}.")}
            m = {k[4:]: t for k, t in w.items() if k.startswith("mix.")}
            L: dict = {}
            for k in (1, 2) if s.has_mlp else (1,):
                pre, post = cfg.norm_names(k)
                L[f"pre{k}"], L[f"post{k}"] = norm(w[pre]) if pre else None, norm(w[post]) if post else None
                if cfg.layer_scale:
                    L[f"post{k}"] *= self._vec(w[f"ls{k}"], dp)
            L["dwa"] = self._vec(w["dwa"]) if cfg.depth_average else None
            if cfg.residual_gate:
                for k in (1, 2) if s.has_mlp else (1,):
                    L[f"rg{k}"], L[f"rg{k}_b"] = self._mat(w[f"rg{k}"], dp, dp), self._vec(w[f"rg{k}.b"], dp)
            getattr(self, "_load_" + s.type)(s, m, L)
            if s.has_mlp:
                getattr(self, "_load_mlp_" + s.mlp)(s, {k[4:]: t for k, t in w.items() if k.startswith("mlp.")}, L)
            self.layers.append(L)
        if cfg.streams:
            self._load_streams(base)

    def _load_streams(self, base: dict[str, torch.Tensor]) -> None:
        """The boundaries of hyper-connected streams.  All copies are equal before the first sublayer and only their sum is read
        behind the last one, so that one copy stands for all at either end."""
        subs = [(i, k) for i, s in enumerate(self.cfg.layers) for k in ((1, 2) if s.has_mlp else (1,))]
        get = lambda i, k, what: base[f"l{i}.hc{k}.{what}"].to(self.device, torch.float64)      # noqa: E731
        for n, (i, k) in enumerate(subs):
            mix, out = get(i, k, "mix"), get(i, k, "out")
            if n == 0:
                mix = mix.sum(0, keepdim=True)
            if n == len(subs) - 1:
                mix, out = mix.sum(1, keepdim=True), out.sum(0, keepdim=True)
                nxt = torch.ones_like(out)
            else:
                nxt = get(*subs[n + 1], "in")
            self.layers[i][f"hc{k}"] = hy.Streams(mix.shape[0], mix.shape[1], torch.cat([mix.flatten(), out, nxt]).float())
        first = get(*subs[0], "in").sum(0, keepdim=True)
        self._embed_streams = hy.Streams(0, 1, torch.cat([torch.ones_like(first), first]).float())

    def _with_gate(self, k: int, W: torch.Tensor, L: dict) -> torch.Tensor:
        """An input matrix with the rows of sublayer ``k``'s residual gate below it; their place is ``L["rg<k>_at"]``."""
        rg = L.pop(f"rg{k}", None)
        if rg is None:
            return W
        L[f"rg{k}_at"] = W.shape[0]
        return torch.cat([W, rg], 0)

    def _gate_of(self, k: int, p: Out, L: dict) -> dict:
        """The residual gate of sublayer ``k`` in its input product's output."""
        at = L.get(f"rg{k}_at")
        return {} if at is None else dict(col_gate=p.col(at), col_bias=L[f"rg{k}_b"])

    def _rotation(self, s: LayerSpec) -> hy.Rotation:
        freq, scale = rope_frequencies(s)
        return hy.Rotation(s.rot_dim, torch.tensor(freq, dtype=torch.float64).to(self.device), scale, s.rot_pairs == "next")

    def _load_latent_attention(self, s: LayerSpec, m: dict, L: dict) -> None:
        rank_p = pad(s.kv_rank, 16)
        L["qkv"] = self._with_gate(1, self._mat(torch.cat([m["q"], m["dkv"]], 0), None, self.dp), L)
        L["sink"] = self._vec(m["sink"]) if s.sink else None
        L["tc_dv"] = hy.prefill_tc_values(s.dim, s.rot_dim, s.vdim, s.scale)
        dk, dv = pad(s.dim, 16), L["tc_dv"] or pad(s.vdim, 16)
        L["c_norm"] = self._vec(m["dkv.norm"])
        uk, uv = m["uk"].view(s.heads, s.dim, s.kv_rank), m["uv"].view(s.heads, s.vdim, s.kv_rank)
        L["uk_t"] = torch.zeros(s.heads, rank_p, pad(s.dim, 16), dtype=self.dtype, device=self.device)
        L["uk_t"][:, :s.kv_rank, :s.dim] = uk.transpose(1, 2).to(self.device)
        L["uv"] = torch.zeros(s.heads, pad(s.vdim), rank_p, dtype=self.dtype, device=self.device)
        L["uv"][:, :s.vdim, :s.kv_rank] = uv.to(self.device)
        if not self.exact32:       # keys of all heads, then values of all heads, from a latent
            kv = torch.zeros(s.heads * (dk + dv), rank_p, dtype=self.dtype, device=self.device)
            kv[:s.heads * dk].view(s.heads, dk, rank_p)[:, :s.dim, :s.kv_rank] = uk.to(self.device)
            kv[s.heads * dk:].view(s.heads, dv, rank_p)[:, :s.vdim, :s.kv_rank] = uv.to(self.device)
            L["ukv"] = kv
        L["rot"] = self._rotation(s)
        L["o"] = self._heads_in(m["o"], s.heads, s.vdim)

    def _load_hgrn2(self, s: LayerSpec, m: dict, L: dict) -> None:
        qv, f = self._mat(torch.cat([m["q"], m["v"]], 0), None, self.dp), self._mat(m["f"], None, self.dp)
        L["qvf"] = torch.cat([qv, f], 0)
        L["qv"], L["f"] = L["qvf"][:qv.shape[0]], L["qvf"][qv.shape[0]:]
        L["f_b"], L["lower"] = self._vec(m["f.b"]), self._vec(m["lower"])
        L["o_norm"] = self._vec(m["norm"])
        L["o"] = self._heads_in(m["o"], s.heads, s.vdim)

    def _load_wkv(self, s: LayerSpec, m: dict, L: dict) -> None:
        n = pad(s.heads * s.dim)
        L["mu"] = torch.stack([self._vec(m["mu." + x], self.dp) for x in SHIFT_MIXES])
        L["rkvg"] = torch.stack([self._mat(m[x], n, self.dp) for x in "rkvg"])
        rp = pad(s.decay_rank)
        L["w1"] = self._mat(m["w1"], rp, self.dp)
        w2 = self._mat(m["w2"], n, rp)
        # bf16: tanh arrives as a pair (high part, remainder), both halves against the same matrix
        L["w2"] = w2 if self.exact32 else torch.cat([w2, w2], 1).contiguous()
        L["w0"], L["u"], L["o_norm"] = self._vec(m["w0"]), self._vec(m["u"]), self._vec(m["norm"])
        L["o"] = self._heads_in(m["o"], s.heads, s.vdim)

    def _load_lightning(self, s: LayerSpec, m: dict, L: dict) -> None:
        L["qkvg"] = self._mat(torch.cat([m["q"], m["k"], m["v"], m["g"]], 0), None, self.dp)
        L["decay"] = torch.tensor(s.decay, dtype=torch.float64).to(self.device, torch.float32)
        L["o_norm"] = self._vec(m["norm"])
        L["o"] = self._heads_in(m["o"], 1, s.heads * s.vdim)

    def _load_parts(self, s: LayerSpec, m: dict, L: dict) -> None:
        """Mixers side by side: their input matrices one below the other (each from a multiple of 8 rows on), their output
        matrices side by side."""
        scales = s.part_scales or (1.0,)
        rows, cols, bias = [], [], torch.zeros(self.dp, dtype=torch.float32, device=self.device)
        L["parts"] = []
        for p, name, scale in zip(s.mixers(), PART_NAMES, scales):
            w = {k[len(name) + 1:]: t for k, t in m.items() if k.startswith(name + ".")} if s.parts else m
            P: dict = {"in": sum(r.shape[0] for r in rows), "out": sum(c.shape[1] for c in cols), "scale": scale}
            r, c = getattr(self, "_load_part_" + p.type)(p, w, P)
            rows.append(r)
            cols.append(c)
            if "o.b" in w:
                bias[:self.cfg.hidden_size] += scale * self._vec(w["o.b"])
            L["parts"].append(P)
        L["in"], L["o"] = self._with_gate(1, torch.cat(rows, 0), L), torch.cat(cols, 1)
        L["o_bias"] = bias if any(p.out_bias for p in s.mixers()) else None

    _load_parallel = _load_attention = _load_rglru = _load_parts

    def _load_part_attention(self, s: LayerSpec, w: dict, P: dict):
        own = "qkv" if s.kv_from < 0 else "q"
        src = self.cfg.layers[s.kv_from] if s.kv_from >= 0 else s
        P["bias"] = self._vec(torch.cat([w[k + ".b"] for k in own])) if s.biases else None
        P["dvp"] = hy.gqa_value_columns(src.dim, src.vdim, src.scale)      # as the cache holds them
        P["tc"] = hy.prefill_tc_values(s.dim, 0, s.vdim, s.scale) == P["dvp"]
        P["kv_heads"] = s.kv_heads if s.kv_from < 0 else 0
        P["q_norm"], P["k_norm"] = (self._vec(w[k + ".norm"]) if s.qk_norm and k in own else None for k in "qk")
        P["temp"] = self._vec(w["temp"]) if s.head_temp else None
        P["table"] = None
        if s.sigmoid:
            P["table"] = hy.distance_table(w["rel"].to(self.device, torch.float32), distance_buckets(s.bias_rows, s.bias_max, s.chunk), self._vec(w["pb"]))
        P["rot"] = self._rotation(s) if s.rot_dim else None
        rows = [w[k] for k in own] + ([w["g"]] if s.head_gate or s.out_gate else [])
        P["g_at"] = sum(r.shape[0] for r in rows) - rows[-1].shape[0] if s.out_gate else 0
        return self._mat(torch.cat(rows, 0), None, self.dp), self._heads_in(w["o"], s.heads, s.vdim)

    def _load_part_rglru(self, s: LayerSpec, w: dict, P: dict):
        n, bp = s.heads * s.dim, pad(s.dim)
        gates = torch.zeros(s.heads, 2, bp, bp, dtype=self.dtype, device=self.device)
        for j, k in enumerate(("ra", "ri")):
            gates[:, j, :s.dim, :s.dim] = w[k].to(self.device)
        gates = gates.view(s.heads, 2 * bp, bp)
        # bf16: the convolution's output arrives as a pair (high part, remainder), both halves against the same matrix
        P["gates"] = gates if self.exact32 else torch.cat([gates, gates], 2).contiguous()
        P["y_b"], P["x_b"], P["r_b"], P["i_b"] = (self._vec(w[k]) for k in ("y.b", "x.b", "ra.b", "ri.b"))
        P["conv"], P["conv_b"] = w["conv"].to(self.device, torch.float32).contiguous(), self._vec(w["conv.b"])
        P["decay"] = (8.0 * torch.nn.functional.softplus(self._vec(w["lam"]).double())).float()
        P["x_col"] = pad(n)
        return torch.cat([self._mat(w["y"], pad(n), self.dp), self._mat(w["x"], pad(n), self.dp)], 0), self._mat(w["o"], self.dp, pad(n))

    def _load_mlp_poly(self, s: LayerSpec, w: dict, L: dict) -> None:
        L["up"], L["down"], L["act"] = self._mat(w["up"], None, self.dp), self._mat(w["down"], self.dp, pad(s.ff)), self._vec(w["act"])

    def _load_mlp_plain(self, s: LayerSpec, w: dict, L: dict) -> None:
        L["up"], L["down"] = self._with_gate(2, self._mat(w["up"], None, self.dp), L), self._mat(w["down"], self.dp, pad(s.ff))

    def _load_mlp_gated(self, s: LayerSpec, w: dict, L: dict) -> None:
        L["gu"], L["down"] = self._glu(w["gate"], w["up"]), self._mat(w["down"], self.dp, pad(s.ff, 16))

    def _load_mlp_moe(self, s: LayerSpec, w: dict, L: dict) -> None:
        ffp = pad(s.expert_ff, 16)

        def inner(name: str, ff: int) -> torch.Tensor:
            return self._glu(w[name + ".gate"], w[name + ".up"]) if s.glu else self._mat(w[name + ".up"], pad(ff, 16), self.dp)

        # the gate of the shared expert is one more row of the router's matrix
        L["router"] = self._with_gate(2, self._mat(torch.cat([w["router"], w["shared.sg"]], 0) if s.shared_gate else w["router"], None, self.dp), L)
        L["router_b"], L["correction"] = (self._vec(w[k]) if k in w else None for k in ("router.b", "correction"))
        n = (2 if s.glu else 1) * ffp
        L["e_in"] = torch.empty(s.experts * n, self.dp, dtype=self.dtype, device=self.device)
        L["e_down"] = torch.empty(s.experts * self.dp, ffp, dtype=self.dtype, device=self.device)
        for e in range(s.experts):
            L["e_in"][e * n:(e + 1) * n] = inner(f"e{e}", s.expert_ff)
            L["e_down"][e * self.dp:(e + 1) * self.dp] = self._mat(w[f"e{e}.down"], self.dp, ffp)
        if s.shared_ff:
            L["s_in"], L["down"] = inner("shared", s.shared_ff), self._mat(w["shared.down"], self.dp, pad(s.shared_ff, 16))

    def set_adapter(self, slot: int, state) -> None:
        if state is not None:
            raise ValueError(f"{self.cfg.name}: adapters are not supported for hybrid models")

    # -- products and buffers -------------------------------------------------------------------------
    def _new(self, M: int, n: int, dtype: torch.dtype | None = None) -> torch.Tensor:
        """An uninitialised [M, n] activation.  The storage of a large batch has its row count rounded up, so that batches
        of nearly the same size ask the allocator for the same blocks."""
        return torch.empty((M if M <= 1024 else pad(M, 1024), n), dtype=dtype or self.dtype, device=self.device)[:M]

    def _mm(self, x, W, f32: bool = False) -> Out:
        out = self._new(x.shape[0], W.shape[0], torch.float32 if f32 else None)
        if self.exact32:
            return as_out(hy.gemm_f32(x, W, out))
        from ..ops.gemm import gemm_tn

        return as_out(gemm_tn(x, W, out=out, out_dtype=out.dtype))

    def _mm_silu(self, x, W, cols: int) -> Out:
        """``x W^T``, the first ``cols`` columns through silu in the product's epilogue (bf16)."""
        from ..ops.gemm import gemm_tn

        return as_out(gemm_tn(x, W, out=self._new(x.shape[0], W.shape[0]), silu_cols=cols))

    def _mm_take(self, b: Ragged, name: str, x, W, f32: bool = False) -> Out:
        """``x W^T`` for a consumer that accepts a split-K workspace: with few rows the product streams the weights from
        all SMs and adds partial sums into the fp32 workspace ``name``, which the consumer reads once and leaves zero."""
        from ..ops.gemm import gemm_splitk_, gemm_tn

        M, N = b.M, W.shape[0]
        bn, splits, pair = self._small_plan(b, W)
        if bn == 0 and not pair:
            return self._mm(x, W, f32)
        if splits == 1:
            return as_out(gemm_tn(x, W, out_dtype=torch.float32 if f32 else torch.bfloat16, bn=bn, two_cta=pair))
        rows = next(n for n in self.BUCKETS if n >= M)
        key = ("ws", name, N, rows)
        ws = self._buf.get(key)
        if ws is None:
            ws = self._buf[key] = torch.zeros((rows, N), dtype=torch.float32, device=self.device)
        gemm_splitk_(ws, x, W, bn, splits, two_cta=bool(pair))
        return Out(ws[:M], hy.KIND_TAKE)

    def _small_plan(self, b: Ragged, W) -> tuple[int, int, bool | None]:
        """``(tile width, splits, CTA pairs)`` of a decode batch's product; ``(0, 1, None)``: the plain product's own choice."""
        from ..ops.gemm import plan_small_m

        M, N, K = b.M, W.shape[0], W.shape[1]
        if not b.single or self.exact32 or M > 512:
            return 0, 1, None
        pair = M % 256 == 0 and N >= 256
        bn, splits = plan_small_m(M, N, K, pair=pair)
        return 0 if pair and splits == 1 else bn, splits, pair

    def _logits(self, hidden) -> torch.Tensor:
        y = self._mm(hidden, self._head, f32=True).t
        return y[:, :self.cfg.vocab_size]

    def _heads_buf(self, name: str, batch: int, M: int, b: Ragged, width: int) -> torch.Tensor:
        """A head-major operand ``[batch, pitch, width]``, row pitch a multiple of 128.  Rows past M are never read back
        but a tile loads them, so the storage starts as zeros and later holds old finite values.  Batches of single
        tokens have buffers of their own size, which stay where they are: captured graphs hold their addresses."""
        pitch = pad(M, 128)
        n = batch * pitch * width
        # one width per buffer: the padding columns of a row are written by nobody
        key = (name, width, n) if b.single else (name, width)
        t = self._buf.get(key)
        if t is None or t.numel() < n or t.device != self.device:
            t = self._buf[key] = torch.zeros(n, dtype=self.dtype, device=self.device)
        return t[:n].view(batch, pitch, width)

    # -- batches ------------------------------------------------------------------------------------------
    def _pack(self, seqs: list[SeqView]) -> tuple[Ragged, list[tuple[int, int]]]:
        """The batch of the sequences' not-yet-cached tokens and, per sequence, its row range."""
        bs, dev = self.kv.shape[1], self.device
        end = [len(s.tokens) if s.upto is None else min(s.upto, len(s.tokens)) for s in seqs]
        order = sorted(range(len(seqs)), key=lambda i: end[i] - seqs[i].num_cached > self.absorb_max)
        portions, n_abs, reach = [], 0, 0
        tok, pos, slot, row_seq, cu, ranges = [], [], [], [], [0], [(0, 0)] * len(seqs)
        for j, i in enumerate(order):
            s = seqs[i]
            n0, n1 = s.num_cached, end[i]
            if n1 <= n0:
                raise ValueError("a scheduled sequence brings at least one token")
            if n1 - n0 <= self.absorb_max:
                n_abs, reach = n_abs + n1 - n0, max(reach, n1)
            else:
                portions.append((j, n0, n1 - n0))
            tok += s.tokens[n0:n1]
            pos += range(n0, n1)
            slot += [s.blocks[t // bs] * bs + t % bs for t in range(n0, n1)]
            row_seq += [j] * (n1 - n0)
            ranges[i] = (cu[-1], cu[-1] + n1 - n0)
            cu.append(cu[-1] + n1 - n0)
        width = max(len(s.blocks) for s in seqs)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)      # noqa: E731
        b = Ragged(cu[-1], len(seqs), torch.tensor(tok, dtype=torch.int64, device=dev), i32(pos), i32(slot), i32(row_seq), i32(cu),
                   i32([end[i] for i in order]), i32([seqs[i].state_slot for i in order]),
                   i32([seqs[i].blocks + [0] * (width - len(seqs[i].blocks)) for i in order]), cu[-1] == len(seqs), portions, n_abs, reach)
        return b, ranges

    # -- layers ---------------------------------------------------------------------------------------------
    def _forward(self, b: Ragged, capture: list | None = None, want_hidden: bool = False):
        """The residual stream ``x`` fp32 [M, dp] behind the last layer and, with ``want_hidden``, its final norm in the
        operand dtype.  ``capture``: receives a copy of the stream after every layer."""
        cfg, dp, d, eps, m = self.cfg, self.dp, self.cfg.hidden_size, self.cfg.norm_eps, self.cfg.residual_mult
        M, dev = b.M, self.device
        x, h = self._new(M, dp, torch.float32), self._new(M, dp)
        wide = self._new(M, cfg.streams * dp, torch.float32) if cfg.streams > 1 else x
        hist = None
        if cfg.depth_average:
            hist = torch.empty((len(self.layers) + 1, M if M <= 1024 else pad(M, 1024), dp), dtype=torch.float32, device=dev)

        def feed(i: int) -> dict:
            """What the stream leaves for layer ``i``'s mixer, or for the output product behind the last layer."""
            if i == len(self.layers):
                return dict(w_next=self.final_norm, h=h) if want_hidden else {}
            return {} if cfg.layers[i].type == "wkv" else dict(w_next=self.layers[i]["pre1"], h=h)      # a token-shift mixer norms its own input

        def boundary(k: int, L: dict, cur, sub: Sublayer, **kw):
            """The stream (or its copies) behind sublayer ``k``."""
            st = L.get(f"hc{k}")
            out = cur if st is None else x if st.n_out == 1 else wide
            hy.residual_step(out, L[f"post{k}"], d, eps, sub=sub, x_in=cur, mult=m, streams=st, **kw)
            return out

        hy.residual_step(x, self.embed_norm, d, eps, mult=cfg.embed_scale, tokens=b.tokens, table=self.embed, freq=self.pos_freq, pos=b.pos,
                         hist=hist, hist_n=0, streams=self._embed_streams if cfg.streams else None, **feed(0))
        cur = x
        for i, (s, L) in enumerate(zip(cfg.layers, self.layers)):
            y, k = getattr(self, "_mix_" + s.type)(i, s, L, cur, h, b), 1
            if s.has_mlp:
                cur = boundary(1, L, cur, y, w_next=L["pre2"], h=h)
                y, k = getattr(self, "_mlp_" + s.mlp)(s, L, cur, h, b), 2
            cur = boundary(k, L, cur, y, hist=hist, hist_n=i + 1, avg=L["dwa"], **feed(i + 1))
            if capture is not None:
                capture.append(cur.view(M, -1, dp)[..., :d].sum(1))
        return cur, h

    # -- feed-forwards ----------------------------------------------------------------------------------------
    def _mlp_poly(self, s: LayerSpec, L, x, h, b: Ragged) -> Sublayer:
        z = self._mm_take(b, "up", h, L["up"])
        a = self._new(b.M, pad(s.ff))
        return Sublayer(self._mm_take(b, "down", hy.poly_norm(z, L["act"], a, s.ff, self.cfg.norm_eps), L["down"]))

    def _glu_product(self, b: Ragged, name: str, h, W, act: str) -> torch.Tensor:
        """``act(h gate^T) * (h up^T)``: the activation in the product's epilogue where the product is not split."""
        a = self._new(b.M, W.shape[0] // 2)
        if not self.exact32 and self._small_plan(b, W)[1] == 1:
            from ..ops.gemm import gemm_tn

            bn, _, pair = self._small_plan(b, W)
            gemm_tn(h, W, swiglu_out=a, gate_act=act, keep_preact=False, bn=bn, two_cta=pair)
            return a
        return hy.gated_act(self._mm_take(b, name, h, W), a, act)

    def _act_product(self, b: Ragged, name: str, h, W, act: str, n: int = 0) -> tuple[torch.Tensor, Out | None]:
        """``act`` of the first ``n`` columns of ``h W^T`` (0: all), likewise, and the product itself where the columns behind them
        are to be taken from."""
        n = n or W.shape[0]
        if not self.exact32 and self._small_plan(b, W)[1] == 1 and act == "relu2":
            from ..ops.gemm import gemm_tn

            bn, _, pair = self._small_plan(b, W)
            z = gemm_tn(h, W, out=self._new(b.M, W.shape[0]), relu2=True, relu2_cols=n, bn=bn, two_cta=pair)
            return z[:, :n], as_out(z)
        z = self._mm_take(b, name, h, W)
        return hy.plain_act(z, self._new(b.M, n), act), z

    def _mlp_plain(self, s: LayerSpec, L, x, h, b: Ragged) -> Sublayer:
        a, z = self._act_product(b, "up", h, L["up"], s.act, pad(s.ff))
        return Sublayer(self._mm_take(b, "down", a, L["down"]), **self._gate_of(2, z, L))

    def _mlp_gated(self, s: LayerSpec, L, x, h, b: Ragged) -> Sublayer:
        return Sublayer(self._mm_take(b, "down", self._glu_product(b, "gu", h, L["gu"], s.act), L["down"]))

    def _mlp_moe(self, s: LayerSpec, L, x, h, b: Ragged) -> Sublayer:
        from ..ops import moe

        z = self._mm_take(b, "router", h, L["router"], f32=True)
        plan = moe.route(z.t[:, :s.experts + s.identity + s.shared_gate], s.top, s.router != "softmax", L["router_b"], take=z.kind == hy.KIND_TAKE,
                         correction=L["correction"], identity=s.identity, gate=s.shared_gate, groups=s.groups, keep=s.group_keep, scale=s.router_scale)
        xp, n, gate = moe.gather(h, plan), L["e_down"].shape[1], self._gate_of(2, z, L)
        a = torch.empty((plan.cap_rows, n), dtype=self.dtype, device=self.device)
        if self.exact32:
            z = as_out(moe.grouped_gemm(xp, L["e_in"], plan, (2 if s.glu else 1) * n))
            (hy.gated_act if s.glu else hy.plain_act)(z, a, s.act)
        elif s.glu:
            moe.grouped_gemm(xp, L["e_in"], plan, 2 * n, swiglu_out=a, keep_preact=False)
        else:
            moe.grouped_gemm(xp, L["e_in"], plan, n, out=a, relu2=True)
        rows = moe.grouped_gemm(a, L["e_down"], plan, self.dp)
        y = None
        if s.shared_ff:
            a = self._glu_product(b, "s_in", h, L["s_in"], s.act) if s.glu else self._act_product(b, "s_in", h, L["s_in"], s.act)[0]
            y = self._mm_take(b, "down", a, L["down"])
        # experts that are the identity take the sublayer's input, in 32-bit where that is the stream itself
        return Sublayer(y, rows=rows, pos=plan.pos, weight=plan.topw, gate=plan.gate,
                        identity=as_out(h if self.cfg.pre_norms else x) if s.identity else None, **gate)

    # -- mixers -------------------------------------------------------------------------------------------------
    def _mix_latent_attention(self, i, s, L, x, h, b: Ragged) -> Sublayer:
        M, H, n_abs = b.M, s.heads, b.n_abs
        cache = self.kv.layers[i]["latent"]
        p = self._mm_take(b, "qkv", h, L["qkv"])
        rank_p, rot_p, dk, dv, vp = pad(s.kv_rank, 16), pad(s.rot_dim, 16), pad(s.dim, 16), pad(s.vdim, 16), pad(s.vdim)
        qn = qr = qe = None
        if n_abs:
            qn, qr = self._heads_buf("qn", H, n_abs, b, dk), self._heads_buf("qr", H, n_abs, b, rot_p)
        if n_abs < M:
            qe = self._new(M - n_abs, H * (dk + rot_p))
        hy.latent_finish(p, L["c_norm"], L["rot"], b.pos, b.slot, cache, n_abs, qn, qr, qe, H, s.dim, s.kv_rank, self.cfg.norm_eps)
        gate, weights = self._gate_of(1, p, L), hy.KeyWeights(sink=L["sink"])
        o = self._new(M, H * vp)
        if n_abs:
            ql, ol = self._heads_buf("ql", H, n_abs, b, rank_p), self._heads_buf("ol", H, n_abs, b, rank_p)
            hy.gemm_batched(qn, L["uk_t"], ql.view(-1, rank_p), n_abs, c_batch=ql.stride(0))
            if self.exact32 or rank_p + rot_p > LATENT_TC_MAX:
                hy.latent_attend(ql, qr, cache, b.bt, b.row_seq, b.pos, b.ctx, s.window, s.scale, ol, n_abs, sink=L["sink"])
            else:
                keys = min(b.reach, s.window) if s.window > 0 else b.reach
                hy.latent_decode(ql, qr, cache, b.bt, b.row_seq, b.pos, b.ctx, s.window, s.scale, ol, n_abs,
                                 hy.latent_decode_splits(n_abs, H, keys), sink=L["sink"])
            hy.gemm_batched(ol, L["uv"], o, n_abs, c_batch=vp)
        if n_abs < M:
            plan = b.plan(s.window)
            c = hy.latent_gather(cache, b.bt, plan)
            if L["tc_dv"]:
                k, vt = self._mm(c[:, :rank_p], L["ukv"][:H * dk]).t, self._mm(L["ukv"][H * dk:], c[:, :rank_p]).t
                hy.latent_prefill_tc(qe, k, vt, c, plan, s.window, s.scale, o[n_abs:], H, dk, L["tc_dv"], rank_p, rot_p, s.vdim, weights=weights)
                return Sublayer(self._mm_take(b, "o", o, L["o"]), **gate)
            kv = self._mm(c[:, :rank_p], L["ukv"]).t
            hy.latent_prefill(qe, kv, c, plan, s.window, s.scale, o[n_abs:], H, dk, dv, rank_p, rot_p, s.vdim, weights=weights)
        return Sublayer(self._mm_take(b, "o", o, L["o"]), **gate)

    def _scan(self, mode, i, s, L, q, k, v, g, aux, bias, gate, b: Ragged) -> Sublayer:
        """Recurrence, per-head norm and gate, output projection."""
        M, H, vp, eps = b.M, s.heads, pad(s.vdim), self.cfg.norm_eps
        state = self.kv.layers[i]["state"]
        per_head = gate is not None
        out = self._new(M, H * vp)
        if b.single:
            hy.linear_decode(mode, q, k, v, g, bias, aux, state, b.cu_q, b.ctx, b.state_slot, H, s.dim, s.vdim, L["o_norm"], per_head,
                             gate, out, vp, eps)
        else:
            o = self._new(M, H * s.vdim, torch.float32)
            hy.linear_scan(mode, q, k, v, g, bias, aux, state, b.cu_q, b.ctx, b.state_slot, b.n_seqs, H, s.dim, s.vdim, o)
            hy.head_norm(o, L["o_norm"], per_head, H, s.vdim, vp, out, eps, gate)
        return Sublayer(self._mm_take(b, "o", out, L["o"]))

    def _mix_hgrn2(self, i, s, L, x, h, b: Ragged) -> Sublayer:
        if b.single:        # one product, its outputs are taken where they lie
            p = self._mm_take(b, "qvf", h, L["qvf"], f32=True)
            qv, g = p, p.col(L["qv"].shape[0])
        else:
            qv, g = self._mm(h, L["qv"]), self._mm(h, L["f"], f32=True)
        return self._scan(hy.SCAN_HGRN2, i, s, L, qv, None, qv.col(s.heads * s.dim), g, L["lower"], L["f_b"], None, b)

    def _mix_wkv(self, i, s, L, x, h, b: Ragged) -> Sublayer:
        M, n = b.M, L["rkvg"].shape[1]
        mixes = self._heads_buf("mix", len(SHIFT_MIXES), M, b, self.dp)
        hy.norm_shift_mix(x, L["pre1"], L["mu"], mixes, self.kv.layers[i]["shift"], b.row_seq, b.cu_q, b.ctx, b.state_slot,
                          self.cfg.hidden_size, self.cfg.norm_eps)
        y = self._new(M, 4 * n)
        if M >= 1024 and not self.exact32:      # four products that each fill the machine: CTA-pair tiles
            from ..ops.gemm import gemm_tn

            for j in range(4):
                gemm_tn(mixes[j, :M], L["rkvg"][j], out=y[:, j * n:(j + 1) * n])
        else:
            hy.gemm_batched(mixes[:4], L["rkvg"], y, M, c_batch=n)
        rp = L["w1"].shape[0]
        z = self._mm_take(b, "w1", mixes[4, :M], L["w1"], f32=True)
        t = self._new(M, L["w2"].shape[1])
        g = self._mm(hy.split_tanh(z, s.decay_rank, rp, t), L["w2"], f32=True)
        y = as_out(y)
        return self._scan(hy.SCAN_WKV, i, s, L, y, y.col(n), y.col(2 * n), g, L["u"], L["w0"], y.col(3 * n), b)

    def _mix_lightning(self, i, s, L, x, h, b: Ragged) -> Sublayer:
        M, n, nv = b.M, s.heads * s.dim, s.heads * s.vdim
        chunked = not b.single and not self.exact32 and hy.lightning_tc(s.dim, s.vdim)
        p = self._mm_silu(h, L["qkvg"], 2 * n + nv) if chunked else self._mm_take(b, "qkvg", h, L["qkvg"])
        q, k, v, gate = p, p.col(n), p.col(2 * n), p.col(2 * n + nv)
        state = self.kv.layers[i]["state"]
        o, out = self._new(M, nv, torch.float32), self._new(M, pad(nv))
        if b.single:
            hy.linear_decode(hy.SCAN_FIXED, q, k, v, None, None, L["decay"], state, b.cu_q, b.ctx, b.state_slot, s.heads, s.dim, s.vdim, None, False,
                             None, o, s.vdim, 0.0)
        elif chunked:
            hy.lightning_prefill(q.t, k.t, v.t, L["decay"], state, b.cu_q, b.ctx, b.state_slot, b.n_seqs, s.heads, s.dim, s.vdim, o)
        else:
            hy.linear_scan(hy.SCAN_FIXED, q, k, v, None, None, L["decay"], state, b.cu_q, b.ctx, b.state_slot, b.n_seqs, s.heads, s.dim, s.vdim, o)
        hy.head_norm(o, L["o_norm"], False, 1, nv, pad(nv), out, self.cfg.norm_eps, gate, hy.GATE_SIGMOID)
        return Sublayer(self._mm_take(b, "o", out, L["o"]))

    def _mix_parts(self, i, s, L, x, h, b: Ragged) -> Sublayer:
        p = self._mm_take(b, "in", h, L["in"])
        o = self._new(b.M, L["o"].shape[1])
        for j, (spec, P) in enumerate(zip(s.mixers(), L["parts"])):
            getattr(self, "_part_" + spec.type)(i, spec, P, p.col(P["in"]), o[:, P["out"]:], self.kv.part(i, j), b)
        return Sublayer(self._mm_take(b, "o", o, L["o"]), bias=L["o_bias"], **self._gate_of(1, p, L))

    _mix_parallel = _mix_attention = _mix_rglru = _mix_parts

    def _part_attention(self, i, s: LayerSpec, P, p: Out, o, cache, b: Ragged) -> None:
        M, n_abs, kv = b.M, b.n_abs, cache["kv"]
        H, G, dk, dvp = s.heads, s.heads // s.kv_heads, pad(s.dim, 16), P["dvp"]
        q, gate, cols, weights = self._new(M, H * dk), None, None, None
        if s.out_gate:                       # the gate's logits stay in the projection, or leave its workspace with the rest
            cols = self._new(M, H * pad(s.vdim)) if p.kind == hy.KIND_TAKE else None
            weights = hy.KeyWeights(P["table"], cols=p.t[:, P["g_at"]:P["g_at"] + H * s.vdim] if cols is None else cols, pitch=s.vdim if cols is None else pad(s.vdim))
        elif s.sigmoid:
            weights = hy.KeyWeights(P["table"])
        if s.out_gate or s.qk_norm or P["rot"] or s.head_gate or s.kv_from >= 0:
            gate = torch.empty((M, H), dtype=torch.float32, device=self.device) if s.head_gate else None
            hy.gqa_finish_norm(p, P["bias"], b.slot, kv, q, H, P["kv_heads"], s.dim, s.vdim, dvp, P["q_norm"], P["k_norm"], self.cfg.norm_eps, P["rot"],
                               b.pos, gate, s.qk_norm_heads, P["temp"], cols, pad(s.vdim) if cols is not None else 0)
        else:
            hy.gqa_finish(p, P["bias"], b.slot, kv, q, H, s.kv_heads, s.dim, s.vdim, dvp)
        if n_abs:
            args = (q, kv, b.bt, b.row_seq, b.pos, b.ctx, s.window, s.chunk, s.scale, P["scale"], o, n_abs, H, s.kv_heads, s.dim, s.vdim, dvp)
            if self.exact32 or max(dk, dvp) > hy.GQA_DECODE_MAX:
                hy.gqa_attend(*args, softcap=s.softcap, gate=gate, weights=weights)
            else:
                reach = min([b.reach] + [w for w in (s.window, s.chunk) if w > 0])
                hy.gqa_decode(*args, splits=hy.gqa_decode_splits(n_abs, s.kv_heads * ((G + 15) // 16), reach), softcap=s.softcap, gate=gate,
                              weights=weights)
        if n_abs < M:
            plan = b.plan(s.window, s.chunk)
            rest = dict(chunk=s.chunk, G=G, out_scale=P["scale"], softcap=s.softcap, gate=gate[n_abs:] if gate is not None else None,
                        weights=weights.rows_from(n_abs) if weights is not None else None)
            src = self.cfg.kv_layer(i)
            key = (src, s.window, s.chunk, P["tc"])
            got = b.kept.get(key)
            if got is None:
                got = hy.gqa_gather(kv, b.bt, plan, s.kv_heads, dk, dvp) if P["tc"] else hy.latent_gather(kv, b.bt, plan)
                if src in self.shared_kv:
                    b.kept[key] = got
            if P["tc"]:
                k, vt = got
                hy.latent_prefill_tc(q[n_abs:], k, vt, k, plan, s.window, s.scale, o[n_abs:], H, dk, dvp, 0, 0, s.vdim, **rest)
            else:
                hy.latent_prefill(q[n_abs:], got, got, plan, s.window, s.scale, o[n_abs:], H, dk, dvp, 0, 0, s.vdim, **rest)

    def _part_rglru(self, i, s: LayerSpec, P, p: Out, o, cache, b: Ragged) -> None:
        M, bp = b.M, pad(s.dim)
        # a buffer of its own per block size: padding columns are written by nobody
        u = self._heads_buf(f"u{s.dim}", s.heads, M, b, P["gates"].shape[2])
        hy.short_conv(p.col(P["x_col"]), P["x_b"], P["conv"], P["conv_b"], cache["conv"], b.row_seq, b.cu_q, b.ctx, b.state_slot, b.n_seqs,
                      b.single, u, s.dim, bp)
        z = self._new(M, s.heads * 2 * bp, torch.float32)
        hy.gemm_batched(u, P["gates"], z, M, c_batch=2 * bp)
        n = s.heads * s.dim
        if n % 8:      # columns between this part and the next: zero weights, but they must be numbers
            o[:, n:pad(n)].zero_()
        hy.rglru(u, z, P["r_b"], P["i_b"], P["decay"], p, P["y_b"], cache["state"], b.cu_q, b.ctx, b.state_slot, b.n_seqs, b.single, o, P["scale"],
                 s.dim, bp)

    # -- the shared loops' hooks ------------------------------------------------------------------------------
    def _prompt_forward(self, seqs: list[SeqView], write_kv: bool = True):
        b, ranges = self._pack(seqs)
        return self._forward(b)[0], ranges

    def layer_outputs(self, seqs: list[SeqView]) -> list[torch.Tensor]:
        """Residual stream after every layer for the sequences' new tokens (rows in batch order); advances their state."""
        out: list[torch.Tensor] = []
        self._forward(self._pack(seqs)[0], capture=out)
        return out

    def _hidden_rows(self, x, rows):
        h = self._new(rows.numel(), self.dp)
        return hy.gather_norm(x, rows, self.final_norm, h, self.cfg.hidden_size, self.cfg.norm_eps)

    def score_view(self, view: SeqView, n_prompt: int) -> list[float]:
        """Log-probabilities of ``view.tokens[n_prompt:]``; the view's blocks and state slot are used as scratch."""
        x, _ = self._prompt_forward([view])
        rows = torch.arange(n_prompt - 1, len(view.tokens) - 1, dtype=torch.int64, device=self.device)
        tgt = torch.tensor(view.tokens[n_prompt:], dtype=torch.int32, device=self.device)
        h = self._hidden_rows(x, rows)
        if self.exact32:
            lp = torch.log_softmax(self._logits(h), -1)
            return lp.gather(-1, tgt.long().unsqueeze(-1)).squeeze(-1).tolist()
        from ..ops import logprob_loss as lpl

        return lpl.grpo_tokens(lpl.partials(h, self.lm_head, tgt)[0]).logprobs.tolist()

    def _decode_buffers(self, nb: int) -> dict:
        dev = self.device
        return {"row_seq": torch.arange(nb, dtype=torch.int32, device=dev), "cu_q": torch.arange(nb + 1, dtype=torch.int32, device=dev),
                "state_slot": torch.full((nb,), -1, dtype=torch.int32, device=dev)}

    def _stage_sequences(self, st, seqs, nb: int) -> None:
        st["state_slot"].copy_(torch.tensor([s.state_slot for s in seqs] + [-1] * (nb - len(seqs)), dtype=torch.int32), non_blocking=True)

    def _attn_splits(self, nb: int, max_ctx: int) -> int:
        """Stands for how far the batch's tokens reach back (a power of two): the attention layers plan their splits by it.
        Contexts beyond every window and chunk change nothing, so that they share one captured graph."""
        windows = [s.window or s.chunk for L in self.cfg.layers for s in L.mixers() if s.type in ("latent_attention", "attention")]
        if not windows:
            return 1
        bound = max_ctx if any(w <= 0 for w in windows) else min(max_ctx, max(windows))
        return 1 << max(0, bound - 1).bit_length()

    def _attn_workspace(self, nb: int, splits: int) -> None:
        return None

    def drop_graphs(self) -> None:
        super().drop_graphs()
        self._buf.clear()         # workspaces of an interrupted step may hold partial sums

    def _decode_steps(self, st, n_steps: int, any_lora: bool, splits: int, ws, restricted: bool, procs) -> None:
        from ..ops import paged

        nb = st["tokens"].shape[0]
        b = Ragged(nb, nb, st["tokens"], st["pos"], st["slot"], st["row_seq"], st["cu_q"], st["ctx"], st["state_slot"], st["bt"], True,
                   n_abs=nb, reach=splits)
        for k in range(n_steps):
            _, hidden = self._forward(b, want_hidden=True)
            t, lp = self._sample(hidden, st["inv_t"], st["seeds"][k], restricted, st["top_k"], st["top_p"], st["min_p"], procs=procs)
            st["out_t"][k].copy_(t)
            st["out_l"][k].copy_(lp)
            if k + 1 < n_steps:
                paged.decode_advance(t, st["tokens"], st["pos"], st["ctx"], st["slot"], st["bt"], self.kv.shape[1], st["active"])
