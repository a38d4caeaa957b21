"""Throughput of hybrid decoders beside the closest Hugging Face family at equal size (``bench.py --hybrid``).

Two parts, random weights throughout:

* ``engine_rows``: prefill and decode tokens/s of whole models through :class:`~art_b200.engine.engine.Engine`, a hybrid
  preset and a twin of the same width, depth and feed-forward parameters per layer, no adapters: a dense Llama-style model,
  or a Qwen3-style mixture of experts where the preset has experts.
* ``kernel_rows``, ``naselorn_kernel_rows``, ``gaborax_kernel_rows``, ``gaparax_kernel_rows``: every kernel of the hybrid path at the
  layer sizes of a model, timed alone with CUDA events (L2 flushed between calls), with its algorithmic bytes and FLOPs and the fraction of its roofline (the slower of bytes at the
  measured copy bandwidth and FLOPs at the measured tensor or nominal fp32 rate), and the like kernels of the dense model
  or of the other design.
"""
from __future__ import annotations

import argparse
import json
import os

import torch

FP32_TFLOPS = 74.4       # nominal: 148 SMs x 128 lanes x 2 x 1.965 GHz


def peaks() -> tuple[float, float]:
    """(GB/s, TFLOP/s bf16) measured on this hardware when the record is there, else earlier figures."""
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            d = json.load(f)
        return float(d["hbm_gbs"]), float(d["bf16_tflops"])
    except (OSError, KeyError, ValueError):
        return 6650.0, 1590.0


def twin(cfg):
    """A Llama-style dense model of the same width and depth whose feed-forward (three matrices) has the hybrid's
    parameters (two matrices), or a Qwen3-style mixture of experts whose experts stand for the hybrid's shared one, too
    (experts of two matrices count as gated ones of two thirds the width)."""
    from ..models.config import ModelConfig

    d = cfg.hidden_size
    moe = next((s for s in cfg.layers if s.experts), None)
    if moe is not None:
        extra = moe.shared_ff // moe.expert_ff
        return ModelConfig(name=f"moe-{cfg.name}", family="qwen3_moe", vocab_size=cfg.vocab_size, hidden_size=d, num_layers=cfg.num_layers,
                           num_heads=d // 128, num_kv_heads=max(1, d // 128 // 4), head_dim=128, intermediate_size=0, qkv_bias=False, qk_norm=True,
                           num_experts=moe.experts + extra, num_experts_per_tok=moe.top + extra, moe_intermediate_size=moe.expert_ff if moe.glu else (moe.expert_ff * 2 // 3 + 15) // 16 * 16)
    ff = max(s.ff for s in cfg.layers)
    return ModelConfig(name=f"dense-{cfg.name}", family="llama", vocab_size=cfg.vocab_size, hidden_size=d, num_layers=cfg.num_layers,
                       num_heads=d // 128, num_kv_heads=max(1, d // 128 // 4), head_dim=128, intermediate_size=(ff * 2 // 3 + 127) // 128 * 128,
                       qkv_bias=False, rope_theta=5e5)


def engine_rows(names: list[str], batches: list[int], prompt_len: int = 1024, new_tokens: int = 64, layers: int = 0):
    from ..models.config import resolve_config
    from .bench_decode import measure_decode

    for name in names:
        cfg = resolve_config(name)
        if layers:
            cfg.layers = cfg.layers[:layers]
        for seqs in batches:
            for c in (cfg, twin(cfg)):
                r = measure_decode(c, "cuda", seqs=seqs, prompt_len=prompt_len, new_tokens=new_tokens, loras=0, prefill_runs=7)
                torch.cuda.empty_cache()
                yield {"model": r["model"], "layers": c.num_layers, "params_b": round(c.num_params() / 1e9, 2), "seqs": seqs,
                       "prompt_len": prompt_len, "new_tokens": new_tokens, "prefill_tok_s": r["prefill_tok_s"],
                       "decode_tok_s": r["decode_tok_s"], "decode_ms_per_step": r["decode_ms_per_step"]}


def _time(fn, flush: torch.Tensor, reps: int = 12) -> float:
    """Median device time of one call in microseconds, L2 flushed before each."""
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    ts = []
    for _ in range(reps):
        flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b) * 1e3)
    return sorted(ts)[len(ts) // 2]


class _Rows:
    """Timed kernels of one layer size."""

    def __init__(self):
        self.gbs, self.tf = peaks()
        self.flush = torch.empty(64 << 20, dtype=torch.float32, device="cuda")
        self.rows: list[dict] = []

    def add(self, name: str, phase: str, fn, bytes_: float, tc_flops: float = 0.0, f32_flops: float = 0.0) -> None:
        us = _time(fn, self.flush)
        floor = max(bytes_ / self.gbs / 1e3, tc_flops / self.tf / 1e6, f32_flops / FP32_TFLOPS / 1e6)
        self.rows.append({"kernel": name, "phase": phase, "us": round(us, 1), "floor_us": round(floor, 1), "of_roofline": round(floor / us, 3),
                          "gb_s": round(bytes_ / us / 1e3, 0), "tflop_s": round((tc_flops + f32_flops) / us / 1e6, 1)})


def kernel_rows(width: int = 4096, ff: int = 16384, prefill: int = 8192, decode: int = 256, window: int = 1024, ctx: int = 2048,
                hist: int = 16) -> list[dict]:
    from ..ops import attention as attn_ops
    from ..ops import elementwise as ew
    from ..ops import hybrid as hy
    from ..ops import paged
    from ..ops.gemm import gemm_tn

    dev, bf = "cuda", torch.bfloat16
    bench = _Rows()
    rows, add = bench.rows, bench.add
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dt=bf, sc=1.0: (torch.randn(*s, device=dev, generator=g) * sc).to(dt)      # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)      # noqa: E731

    d = width
    for phase, M in (("decode", decode), ("prefill", prefill)):
        one = phase == "decode"
        n_seqs = M if one else M // 2048
        cu = i32(list(range(M + 1)) if one else [i * 2048 for i in range(n_seqs + 1)])
        row_seq = i32(list(range(M)) if one else [i // 2048 for i in range(M)])
        c_len = i32([ctx] * n_seqs)
        pos = i32([ctx - 1] * M if one else [i % 2048 for i in range(M)])
        slots = i32(list(range(n_seqs)))
        x, w, h = rnd(M, d, dt=torch.float32), rnd(d, dt=torch.float32), rnd(M, d)
        y = rnd(M, d)
        add("residual_step", phase, lambda: hy.residual_step(x, w, d, 1e-5, y=hy.as_out(y), x_in=x, mult=0.5, w_next=w, h=h), M * d * 12)
        hs = rnd(hist + 1, M, d, dt=torch.float32)
        avg = rnd(hist + 1, dt=torch.float32, sc=0.1)
        add(f"residual_step, average of {hist}", phase, lambda: hy.residual_step(x, w, d, 1e-5, y=hy.as_out(y), x_in=x, mult=0.5, hist=hs,
                                                                             hist_n=hist, avg=avg, w_next=w, h=h), M * d * (16 + 4 * hist))
        add("like: rmsnorm_fwd (bf16)", phase, lambda: ew.rmsnorm_fwd(y, w.to(bf), 1e-5, want_rstd=False), M * d * 4)
        del hs
        shift, mu = rnd(n_seqs, d, dt=torch.float32), rnd(5, d, dt=torch.float32)
        mixes = torch.zeros(5, hy.pad(M, 128), d, dtype=bf, device=dev)
        add("norm_shift_mix", phase, lambda: hy.norm_shift_mix(x, w, mu, mixes, shift, row_seq, cu, c_len, slots, d, 1e-5), M * d * 14)
        W4 = rnd(4, d, d, sc=d ** -0.5)
        y4 = torch.empty(M, 4 * d, dtype=bf, device=dev)
        add("gemm_batched r|k|v|g", phase, lambda: hy.gemm_batched(mixes[:4], W4, y4, M, c_batch=d), (4 * d * d + 8 * M * d) * 2, 8.0 * M * d * d)
        wq = W4.view(4 * d, d)
        add("like: gemm_tn, same product size", phase, lambda: gemm_tn(y, wq), (4 * d * d + 5 * M * d) * 2, 8.0 * M * d * d)
        z, act = rnd(M, ff), rnd(4, dt=torch.float32)
        out = torch.empty_like(z)
        add("poly_norm", phase, lambda: hy.poly_norm(hy.as_out(z), act, out, ff, 1e-5), M * ff * 4)
        del z, out
        # linear attention
        for mode, name, H, dim in ((hy.SCAN_HGRN2, "hgrn2", d // 128, 128), (hy.SCAN_WKV, "wkv", d // 64, 64)):
            n = H * dim
            st = torch.zeros(n_seqs, H, dim, dim, dtype=torch.float32, device=dev)
            q, gr = rnd(M, 4 * n), rnd(M, n, dt=torch.float32)
            aux = torch.rand(n, device=dev, generator=g)
            Q = hy.as_out(q)
            k = Q.col(n) if mode == hy.SCAN_WKV else None
            gate = Q.col(3 * n) if mode == hy.SCAN_WKV else None
            nw = rnd(n if gate else dim, dt=torch.float32)
            o16 = torch.empty(M, n, dtype=bf, device=dev)
            in_bytes = M * n * (2 * (3 if k else 2) + 4)
            flops = M * H * dim * dim * (5.0 if mode == hy.SCAN_WKV else 5.0)
            if one:
                add(f"linear_decode {name} {H} x {dim}^2", phase, lambda: hy.linear_decode(
                    mode, Q, k, Q.col(2 * n), hy.as_out(gr), aux, aux, st, cu, c_len, slots, H, dim, dim, nw, gate is not None, gate, o16, dim, 1e-5),
                    in_bytes + M * n * 2 + 8.0 * st.numel(), f32_flops=flops)
            else:
                o = torch.empty(M, n, dtype=torch.float32, device=dev)
                add(f"linear_scan {name} {H} x {dim}^2", phase, lambda: hy.linear_scan(
                    mode, Q, k, Q.col(2 * n), hy.as_out(gr), aux, aux, st, cu, c_len, slots, n_seqs, H, dim, dim, o),
                    in_bytes + M * n * 4 + 8.0 * st.numel(), f32_flops=flops)
                add(f"head_norm {name}", phase, lambda: hy.head_norm(o, nw, gate is not None, H, dim, dim, o16, 1e-5, gate), M * n * (8 if gate else 6))
        # latent attention: d / 128 heads of 128 + 64, latent 512, values 128
        H, dk, rot, rank, dv, bs = d // 128, 128, 64, 512, 128, 16
        ldc = rank + rot
        nb = n_seqs * (ctx // bs)
        cache = rnd(nb, bs, ldc)
        bt = torch.randperm(nb, device=dev, generator=g).to(torch.int32).view(n_seqs, ctx // bs)
        pq = rnd(M, H * (dk + rot) + rank + rot)
        turn = hy.Rotation(rot, rnd(rot // 2, dt=torch.float64), next=True)
        cn = rnd(rank, dt=torch.float32)
        slot = i32([-1] * M)
        qn, qr = torch.zeros(H, hy.pad(M, 128), dk, dtype=bf, device=dev), torch.zeros(H, hy.pad(M, 128), rot, dtype=bf, device=dev)
        qe = torch.zeros(M, H * (dk + rot), dtype=bf, device=dev)
        add("latent_finish", phase, lambda: hy.latent_finish(hy.as_out(pq), cn, turn, pos, slot, cache, M if one else 0, qn, qr, qe, H, dk, rank, 1e-5),
            M * (2 * H * (dk + rot) + rank + rot) * 2)
        if one:
            ql, ol = rnd(H, hy.pad(M, 128), rank), torch.zeros(H, hy.pad(M, 128), rank, dtype=bf, device=dev)
            sp = hy.latent_decode_splits(M, H, window)
            keys = min(window, ctx)
            add(f"latent_decode window {window}", phase, lambda: hy.latent_decode(ql, qr, cache, bt, row_seq, pos, c_len, window, 0.07, ol, M, sp),
                M * keys * ldc * 2 + M * H * (2 * rank + rot) * 2, 2.0 * M * H * keys * (2 * rank + rot))
            uk = rnd(H, rank, dk, sc=0.05)
            add("gemm_batched q~ (heads)", phase, lambda: hy.gemm_batched(qn, uk, ql.view(-1, rank), M, c_batch=ql.stride(0)),
                H * (rank * dk + M * (rank + dk)) * 2, 2.0 * M * H * rank * dk)
            uv = rnd(H, dv, rank, sc=0.05)
            oo = torch.empty(M, H * dv, dtype=bf, device=dev)
            add("gemm_batched W_uv (heads)", phase, lambda: hy.gemm_batched(ol, uv, oo, M, c_batch=dv), H * (rank * dv + M * (rank + dv)) * 2,
                2.0 * M * H * rank * dv)
            Hkv = max(1, H // 4)
            kc, vc = rnd(n_seqs * window // bs, bs, Hkv, 128), rnd(n_seqs * window // bs, bs, Hkv, 128)
            btd = torch.arange(n_seqs * window // bs, dtype=torch.int32, device=dev).view(n_seqs, -1)
            qd, od = rnd(M, H * 128), torch.empty(M, H * 128, dtype=bf, device=dev)
            cd = i32([window] * M)
            add(f"like: paged_decode ctx {window}", phase, lambda: paged.paged_decode(qd, kc, vc, btd, cd, H, Hkv, 128, od), M * window * Hkv * 512,
                4.0 * M * H * window * 128)
        else:
            plan = hy.plan_prefill([(i, 0, 2048) for i in range(n_seqs)], window, dev)
            c = hy.latent_gather(cache, bt, plan)
            add("latent_gather", phase, lambda: hy.latent_gather(cache, bt, plan), plan.n_keys * ldc * 4)
            kv, o = rnd(plan.n_keys, H * (dk + dv)), torch.empty(M, H * dv, dtype=bf, device=dev)
            pairs = n_seqs * sum(min(i + 1, window) for i in range(2048))
            k, vt = rnd(plan.n_keys, H * dk), rnd(H * dv, plan.n_keys)
            add(f"latent_prefill_tc window {window}", phase, lambda: hy.latent_prefill_tc(qe, k, vt, c, plan, window, 0.07, o, H, dk, dv, rank, rot, dv),
                (qe.numel() + kv.numel() + o.numel()) * 2, 2.0 * H * pairs * (dk + rot + dv))
            add(f"latent_prefill (any sizes) window {window}", phase, lambda: hy.latent_prefill(qe, kv, c, plan, window, 0.07, o, H, dk, dv, rank, rot, dv),
                (qe.numel() + kv.numel() + o.numel()) * 2, 2.0 * H * pairs * (dk + rot + dv))
            ids = torch.arange(n_seqs, dtype=torch.int32, device=dev).repeat_interleave(2048)
            ap = attn_ops.make_plan(ids, ids, M, "native")
            Hkv = max(1, H // 4)
            qkv = rnd(M, (H + 2 * Hkv) * 128)
            add("like: tree attention fwd, causal, head 128", phase, lambda: attn_ops.forward(qkv, H, Hkv, 128, ap, need_grad=False),
                qkv.numel() * 2 + M * H * 256, 4.0 * H * 128 * n_seqs * 2048 * 2049 / 2)
    return rows


def naselorn_kernel_rows(width: int = 4096, prefill: int = 8192, decode: int = 256, chunk: int = 1024, ctx: int = 2048, experts: int = 64,
                         top: int = 8, expert_ff: int = 1024, dense_ff: int = 12288, block: int = 256) -> list[dict]:
    """The kernels of Naselorn layers, each beside the like kernel of another design where there is one ("like: ...")."""
    from ..ops import attention as attn_ops
    from ..ops import elementwise as ew
    from ..ops import hybrid as hy
    from ..ops import moe, paged
    from ..ops.gemm import gemm_tn

    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    bench = _Rows()
    add = bench.add
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dt=bf, sc=1.0: (torch.randn(*s, device=dev, generator=g) * sc).to(dt)      # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)      # noqa: E731
    d, H, hd, bs = width, width // 128, 128, 16
    Hkv, G = H // 4, 4
    for phase, M in (("decode", decode), ("prefill", prefill)):
        one = phase == "decode"
        n_seqs = M if one else M // 2048
        cu = i32(list(range(M + 1)) if one else [i * 2048 for i in range(n_seqs + 1)])
        row_seq = i32(list(range(M)) if one else [i // 2048 for i in range(M)])
        c_len, slots = i32([ctx] * n_seqs), i32(list(range(n_seqs)))
        pos = i32([ctx - 1] * M if one else [i % 2048 for i in range(M)])
        x, w, h, y = rnd(M, d, dt=f32), rnd(d, dt=f32), rnd(M, d), rnd(M, d)
        add("residual_step (pre-norm frame)", phase, lambda: hy.residual_step(x, None, d, 1e-5, y=hy.as_out(y), x_in=x, w_next=w, h=h), M * d * 12)
        add("like: residual_step with post-norm", phase, lambda: hy.residual_step(x, w, d, 1e-5, y=hy.as_out(y), x_in=x, mult=0.5, w_next=w, h=h), M * d * 12)
        # lightning attention
        n = H * hd
        p, st = rnd(M, 4 * n), torch.zeros(n_seqs, H, hd, hd, dtype=f32, device=dev)
        P = hy.as_out(p)
        decay = torch.rand(H, device=dev, generator=g)
        o, o16, nw = torch.empty(M, n, dtype=f32, device=dev), torch.empty(M, n, dtype=bf, device=dev), rnd(n, dt=f32)
        gr, aux = rnd(M, n, dt=f32), torch.rand(n, device=dev, generator=g)
        scan = (decay, st, cu, c_len, slots)
        in_bytes, flops = M * n * 6, 5.0 * M * H * hd * hd
        if one:
            add(f"linear_decode fixed {H} x {hd}^2", phase, lambda: hy.linear_decode(hy.SCAN_FIXED, P, P.col(n), P.col(2 * n), None, None, *scan, H, hd, hd, None,
                                                                                 False, None, o, hd, 0.0), in_bytes + M * n * 4 + 8.0 * st.numel(), f32_flops=flops)
            add(f"like: linear_decode hgrn2 {H} x {hd}^2", phase, lambda: hy.linear_decode(
                hy.SCAN_HGRN2, P, None, P.col(2 * n), hy.as_out(gr), aux, aux, st, cu, c_len, slots, H, hd, hd, nw[:hd], False, None, o16, hd, 1e-5),
                M * n * 10 + 8.0 * st.numel(), f32_flops=flops)
        else:
            # chunked form: q k^T, its product with v, q S and the state's update, the latter two with split operands
            tc = 2.0 * M * H * (64 * hd + 2 * 64 * hd + 4 * hd * hd)
            add(f"lightning_prefill {H} x {hd}^2", phase, lambda: hy.lightning_prefill(p[:, :n], p[:, n:2 * n], p[:, 2 * n:3 * n], *scan, n_seqs, H, hd, hd, o),
                in_bytes + M * n * 4 + 8.0 * st.numel(), tc_flops=tc)
            add(f"linear_scan fixed {H} x {hd}^2 (odd sizes, fp32)", phase, lambda: hy.linear_scan(
                hy.SCAN_FIXED, P, P.col(n), P.col(2 * n), None, None, *scan, n_seqs, H, hd, hd, o), in_bytes + M * n * 4 + 8.0 * st.numel(), f32_flops=flops)
            add(f"like: linear_scan hgrn2 {H} x {hd}^2", phase, lambda: hy.linear_scan(
                hy.SCAN_HGRN2, P, None, P.col(2 * n), hy.as_out(gr), aux, aux, st, cu, c_len, slots, n_seqs, H, hd, hd, o),
                M * n * 12 + 8.0 * st.numel(), f32_flops=flops)
        add("row_norm with sigmoid gate", phase, lambda: hy.head_norm(o, nw, False, 1, n, n, o16, 1e-5, P.col(3 * n), hy.GATE_SIGMOID), M * n * 8)
        add("like: head_norm with silu gate", phase, lambda: hy.head_norm(o, nw, True, H, hd, hd, o16, 1e-5, P.col(3 * n)), M * n * 8)
        del st, gr, p, P
        # chunked grouped-query attention
        ld = Hkv * 2 * hd
        nb = n_seqs * (ctx // bs)
        cache = rnd(nb, bs, ld)
        bt = torch.randperm(nb, device=dev, generator=g).to(torch.int32).view(n_seqs, ctx // bs)
        qkv, bias = rnd(M, (H + 2 * Hkv) * hd), rnd((H + 2 * Hkv) * hd, dt=f32)
        q, slot = torch.empty(M, H * hd, dtype=bf, device=dev), i32([i % (nb * bs) for i in range(M)])
        add("gqa_finish", phase, lambda: hy.gqa_finish(hy.as_out(qkv), bias, slot, cache, q, H, Hkv, hd, hd, hd), 2 * qkv.numel() * 2)
        ao = torch.empty(M, H * hd, dtype=bf, device=dev)
        if one:
            sp = hy.gqa_decode_splits(M, Hkv, chunk)
            keys = (ctx - 1) % chunk + 1
            add(f"gqa_decode chunk {chunk}", phase, lambda: hy.gqa_decode(q, cache, bt, row_seq, pos, c_len, 0, chunk, hd ** -0.5, 0.5, ao, M, H, Hkv, hd, hd, hd, sp),
                M * keys * ld * 2 + M * H * hd * 4, 4.0 * M * H * keys * hd)
            kc, vc = rnd(n_seqs * chunk // bs, bs, Hkv, hd), rnd(n_seqs * chunk // bs, bs, Hkv, hd)
            btd = torch.arange(n_seqs * chunk // bs, dtype=torch.int32, device=dev).view(n_seqs, -1)
            cd = i32([chunk] * M)
            add(f"like: paged_decode ctx {chunk}", phase, lambda: paged.paged_decode(q, kc, vc, btd, cd, H, Hkv, hd, ao), M * chunk * ld * 2 + M * H * hd * 4,
                4.0 * M * H * chunk * hd)
        else:
            plan = hy.plan_prefill([(i, 0, 2048) for i in range(n_seqs)], 0, dev, chunk)
            add("gqa_gather", phase, lambda: hy.gqa_gather(cache, bt, plan, Hkv, hd, hd), plan.n_keys * ld * 4)
            add("like: latent_gather", phase, lambda: hy.latent_gather(cache, bt, plan), plan.n_keys * ld * 4)
            k, vt = hy.gqa_gather(cache, bt, plan, Hkv, hd, hd)
            pairs = n_seqs * sum(i % chunk + 1 for i in range(2048))
            add(f"latent_prefill_tc chunk {chunk}", phase, lambda: hy.latent_prefill_tc(q, k, vt, k, plan, 0, hd ** -0.5, ao, H, hd, hd, 0, 0, hd, chunk=chunk, G=G),
                (q.numel() + k.numel() + vt.numel() + ao.numel()) * 2, 4.0 * H * pairs * hd)
            ids = torch.arange(M // chunk, dtype=torch.int32, device=dev).repeat_interleave(chunk)
            ap = attn_ops.make_plan(ids, ids, M, "native")
            add(f"like: tree attention fwd, causal, {chunk} tokens", phase, lambda: attn_ops.forward(qkv, H, Hkv, hd, ap, need_grad=False),
                qkv.numel() * 2 + M * H * hd * 2, 4.0 * H * pairs * hd)
        # gated linear recurrent unit
        nblk, bp = d // block, block
        xy = hy.as_out(rnd(M, 2 * d))
        u = torch.zeros(nblk, hy.pad(M, 128), 2 * bp, dtype=bf, device=dev)
        cw, cst, rst = rnd(d, 4, dt=f32), torch.zeros(n_seqs, 3, d, device=dev), torch.zeros(n_seqs, d, device=dev)
        add("short_conv", phase, lambda: hy.short_conv(xy.col(d), w, cw, w, cst, row_seq, cu, c_len, slots, n_seqs, one, u, block, bp), M * d * 6 + cst.numel() * 8)
        gates, z = rnd(nblk, 2 * bp, 2 * bp, sc=block ** -0.5), torch.empty(M, 2 * d, dtype=f32, device=dev)
        add("gemm_batched gates", phase, lambda: hy.gemm_batched(u, gates, z, M, c_batch=2 * bp), gates.numel() * 2 + M * d * 12, 2.0 * M * d * 4 * bp)
        dec = torch.rand(d, device=dev, generator=g)
        add("rglru", phase, lambda: hy.rglru(u, z, w, w, dec, xy, w, rst, cu, c_len, slots, n_seqs, one, o16, 0.5, block, bp), M * d * 16 + rst.numel() * 8)
        del u, z, xy
        # feed-forwards
        gu = rnd(M, 2 * dense_ff)
        a = torch.empty(M, dense_ff, dtype=bf, device=dev)
        add("gated_act", phase, lambda: hy.gated_act(hy.as_out(gu), a, "relu"), M * dense_ff * 6)
        add("like: swiglu_fwd", phase, lambda: ew.swiglu_fwd(gu, out=a), M * dense_ff * 6)
        Wg = rnd(2 * dense_ff, d, sc=d ** -0.5)
        pf = 4.0 * M * d * dense_ff
        if not one:
            add("gemm_tn gate|up, relu epilogue", phase, lambda: gemm_tn(h, Wg, swiglu_out=a, gate_act="relu", keep_preact=False),
                (Wg.numel() + M * d + a.numel()) * 2, pf)
            add("like: gemm_tn gate|up, silu epilogue", phase, lambda: gemm_tn(h, Wg, out=gu, swiglu_out=a), (Wg.numel() + M * d + 3 * a.numel()) * 2, pf)
            Wp, qp = Wg[:4 * n], torch.empty(M, 4 * n, dtype=bf, device=dev)
            qf = 2.0 * M * d * 4 * n
            add("gemm_tn q|k|v|g, silu epilogue", phase, lambda: gemm_tn(h, Wp, out=qp, silu_cols=3 * n), (Wp.numel() + M * d + qp.numel()) * 2, qf)
            add("like: gemm_tn, same product", phase, lambda: gemm_tn(h, Wp, out=qp), (Wp.numel() + M * d + qp.numel()) * 2, qf)
            del qp, Wp
        del gu, a, Wg
        logits, rb = rnd(M, experts, dt=f32), rnd(experts, dt=f32)
        add("moe.route (router, plan)", phase, lambda: moe.route(logits, top, True, rb), M * (experts * 4 + top * 8))
        add("like: moe.route without bias", phase, lambda: moe.route(logits, top, True), M * (experts * 4 + top * 8))
        rp = moe.route(logits, top, True, rb)
        xp = moe.gather(h, rp)
        add("moe.gather", phase, lambda: moe.gather(h, rp, out=xp), M * d * 2 * (1 + top))
        eg, ed = rnd(experts * 2 * expert_ff, d, sc=d ** -0.5), rnd(experts * d, expert_ff, sc=expert_ff ** -0.5)
        ea = torch.empty(rp.cap_rows, expert_ff, dtype=bf, device=dev)
        yp = torch.empty(rp.cap_rows, d, dtype=bf, device=dev)
        ef = 2.0 * M * top * d * expert_ff
        add("grouped_gemm gate|up, silu epilogue", phase, lambda: moe.grouped_gemm(xp, eg, rp, 2 * expert_ff, swiglu_out=ea, keep_preact=False),
            (eg.numel() + M * top * (d + expert_ff)) * 2, 2 * ef)
        add("grouped_gemm down", phase, lambda: moe.grouped_gemm(ea, ed, rp, d, out=yp), (ed.numel() + M * top * (d + expert_ff)) * 2, ef)
        sub = hy.Sublayer(hy.as_out(y), rows=yp, pos=rp.pos, weight=rp.topw)
        add("residual_step with experts' rows", phase, lambda: hy.residual_step(x, None, d, 1e-5, sub=sub, x_in=x, w_next=w, h=h), M * d * (12 + 2 * top))
        add("like: moe.combine", phase, lambda: moe.combine(yp, rp, residual=y), M * d * 2 * (2 + top))
        del eg, ed, ea, yp, xp, cache, qkv, q, ao, o, o16
        torch.cuda.empty_cache()
    return bench.rows


def gaborax_kernel_rows(width: int = 4096, prefill: int = 8192, decode: int = 256, ctx: int = 2048, experts: int = 64, identity: int = 8,
                        top: int = 8, expert_ff: int = 1536, shared_ff: int = 3072, softcap: float = 50.0) -> list[dict]:
    """The kernels of Gaborax layers, each beside the like kernel of another design ("like: ...")."""
    from ..ops import attention as attn_ops
    from ..ops import hybrid as hy
    from ..ops import moe, paged
    from ..ops.gemm import gemm_tn

    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    bench = _Rows()
    add = bench.add
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dt=bf, sc=1.0: (torch.randn(*s, device=dev, generator=g) * sc).to(dt)      # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)      # noqa: E731
    d, H, hd, bs = width, width // 128, 128, 16
    Hkv, G = H // 4, 4
    freq = torch.tensor([5e5 ** (-2 * i / hd) for i in range(hd // 2)], dtype=torch.float64, device=dev)
    for phase, M in (("decode", decode), ("prefill", prefill)):
        one = phase == "decode"
        n_seqs = M if one else M // 2048
        row_seq = i32(list(range(M)) if one else [i // 2048 for i in range(M)])
        c_len = i32([ctx] * n_seqs)
        pos = i32([ctx - 1] * M if one else [i % 2048 for i in range(M)])
        x, w, h, y = rnd(M, d, dt=f32), rnd(d, dt=f32), rnd(M, d), rnd(M, d)
        add("residual_step, post-norm, stream as operand", phase, lambda: hy.residual_step(x, w, d, 1e-5, y=hy.as_out(y), x_in=x, h=h), M * d * 12)
        add("like: residual_step with both norms", phase, lambda: hy.residual_step(x, w, d, 1e-5, y=hy.as_out(y), x_in=x, w_next=w, h=h), M * d * 12)
        # attention
        ld = Hkv * 2 * hd
        nb = n_seqs * (ctx // bs)
        cache = rnd(nb, bs, ld)
        bt = torch.randperm(nb, device=dev, generator=g).to(torch.int32).view(n_seqs, ctx // bs)
        n = (H + 2 * Hkv) * hd
        qkvg, bias, wn = rnd(M, n + H), rnd(n, dt=f32), rnd(n, dt=f32)
        q, slot = torch.empty(M, H * hd, dtype=bf, device=dev), i32([i % (nb * bs) for i in range(M)])
        gate = torch.empty(M, H, dtype=f32, device=dev)
        P = hy.as_out(qkvg)
        for nxt, gt, b_ in ((False, gate, None), (True, None, bias)):
            add("gqa_finish_norm, " + ("neighbours, biases" if nxt else "halves, gates"), phase, lambda: hy.gqa_finish_norm(
                P, b_, slot, cache, q, H, Hkv, hd, hd, hd, wn, wn, 1e-5, hy.Rotation(hd, freq, 1.1, nxt), pos, gt), M * n * 4)
        add("gqa_finish_norm, queries alone", phase, lambda: hy.gqa_finish_norm(P, None, slot, cache, q, H, 0, hd, hd, hd, wn, None, 1e-5, hy.Rotation(hd, freq), pos, gate),
            M * H * hd * 4)
        add("like: gqa_finish (no norm, no rotation)", phase, lambda: hy.gqa_finish(P, bias, slot, cache, q, H, Hkv, hd, hd, hd), M * n * 4)
        ao = torch.empty(M, H * hd, dtype=bf, device=dev)
        forms = (("gate", dict(gate=gate)), (f"softcap {softcap:.0f}", dict(softcap=softcap)))
        if one:
            sp = hy.gqa_decode_splits(M, Hkv, ctx)
            b_, f_ = M * ctx * ld * 2 + M * H * hd * 4, 4.0 * M * H * ctx * hd
            for name, kw in forms:
                add(f"gqa_decode ctx {ctx}, {name}", phase, lambda: hy.gqa_decode(q, cache, bt, row_seq, pos, c_len, 0, 0, hd ** -0.5, 1.0, ao, M, H, Hkv, hd, hd, hd, sp,
                                                                               **kw), b_, f_)
            kc, vc = rnd(nb, bs, Hkv, hd), rnd(nb, bs, Hkv, hd)
            add(f"like: paged_decode ctx {ctx}", phase, lambda: paged.paged_decode(q, kc, vc, bt, c_len, H, Hkv, hd, ao), b_, f_)
            del kc, vc
        else:
            plan = hy.plan_prefill([(i, 0, 2048) for i in range(n_seqs)], 0, dev)
            add("gqa_gather", phase, lambda: hy.gqa_gather(cache, bt, plan, Hkv, hd, hd), plan.n_keys * ld * 4)
            add("like: latent_gather", phase, lambda: hy.latent_gather(cache, bt, plan), plan.n_keys * ld * 4)
            k, vt = hy.gqa_gather(cache, bt, plan, Hkv, hd, hd)
            pairs = n_seqs * 2048 * 2049 // 2
            b_, f_ = (q.numel() + k.numel() + vt.numel() + ao.numel()) * 2, 4.0 * H * pairs * hd
            for name, kw in (("plain", {}),) + forms:
                add(f"latent_prefill_tc causal 2048, {name}", phase, lambda: hy.latent_prefill_tc(q, k, vt, k, plan, 0, hd ** -0.5, ao, H, hd, hd, 0, 0, hd, G=G, **kw), b_, f_)
            c = hy.latent_gather(cache, bt, plan)
            for name, kw in (("plain", {}), forms[1]):
                add(f"latent_prefill (any sizes) causal 2048, {name}", phase, lambda: hy.latent_prefill(q, c, c, plan, 0, hd ** -0.5, ao, H, hd, hd, 0, 0, hd, G=G, **kw), b_, f_)
            ids = torch.arange(n_seqs, dtype=torch.int32, device=dev).repeat_interleave(2048)
            ap = attn_ops.make_plan(ids, ids, M, "native")
            qkv = qkvg[:, :n].contiguous()
            add("like: tree attention fwd, causal, 2048 tokens", phase, lambda: attn_ops.forward(qkv, H, Hkv, hd, ap, need_grad=False), b_, f_)
            del qkv, k, vt, c
        # feed-forward
        a, Wu = torch.empty(M, shared_ff, dtype=bf, device=dev), rnd(shared_ff, d, sc=d ** -0.5)
        wb, wf = (Wu.numel() + M * d + a.numel()) * 2, 2.0 * M * d * shared_ff
        add("gemm_tn up, squared relu epilogue", phase, lambda: gemm_tn(h, Wu, out=a, relu2=True), wb, wf)
        add("like: gemm_tn, same product", phase, lambda: gemm_tn(h, Wu, out=a), wb, wf)
        z = rnd(M, shared_ff, dt=f32)
        add("plain_act (split products)", phase, lambda: hy.plain_act(hy.Out(z, hy.KIND_TAKE), a, "relu2"), M * shared_ff * 10)
        z2 = rnd(M, 2 * shared_ff, dt=f32)
        add("like: gated_act", phase, lambda: hy.gated_act(hy.Out(z2, hy.KIND_TAKE), a, "silu"), M * shared_ff * 18)
        del z, z2, a, Wu
        outputs = experts + identity
        logits, corr = rnd(M, outputs + 1, dt=f32), rnd(outputs, dt=f32, sc=1e-3)
        add("moe.route by corrected scores", phase, lambda: moe.route(logits, top, True, correction=corr, identity=identity, gate=True), M * (outputs * 4 + top * 8))
        add("like: moe.route by logits", phase, lambda: moe.route(logits[:, :experts], top, True, corr), M * (outputs * 4 + top * 8))
        rp = moe.route(logits, top, True, correction=corr, identity=identity, gate=True)
        real = int((rp.topi < experts).sum())
        xp = moe.gather(h, rp)
        add("moe.gather", phase, lambda: moe.gather(h, rp, out=xp), d * 2 * (M + real))
        eu, ed = rnd(experts * expert_ff, d, sc=d ** -0.5), rnd(experts * d, expert_ff, sc=expert_ff ** -0.5)
        ea, yp = torch.empty(rp.cap_rows, expert_ff, dtype=bf, device=dev), torch.empty(rp.cap_rows, d, dtype=bf, device=dev)
        eb, ef = (eu.numel() + real * (d + expert_ff)) * 2, 2.0 * real * d * expert_ff
        add("grouped_gemm up, squared relu epilogue", phase, lambda: moe.grouped_gemm(xp, eu, rp, expert_ff, out=ea, relu2=True), eb, ef)
        eg = eu[:experts * (expert_ff // 32 * 32)]
        sw = torch.empty(rp.cap_rows, expert_ff // 2, dtype=bf, device=dev)
        add("like: grouped_gemm gate|up, silu epilogue, same product", phase, lambda: moe.grouped_gemm(xp, eg, rp, expert_ff, swiglu_out=sw, keep_preact=False),
            (eu.numel() + real * (d + expert_ff // 2)) * 2, ef)
        add("grouped_gemm down", phase, lambda: moe.grouped_gemm(ea, ed, rp, d, out=yp), eb, ef)
        sub = hy.Sublayer(hy.as_out(y), rows=yp, pos=rp.pos, weight=rp.topw, gate=rp.gate, identity=hy.as_out(x))
        add("residual_step with experts' rows, gate, identity", phase, lambda: hy.residual_step(x, w, d, 1e-5, sub=sub, x_in=x, h=h), M * d * 12 + real * d * 2)
        plain = hy.Sublayer(hy.as_out(y), rows=yp, pos=rp.pos.clamp(min=0), weight=rp.topw)
        add("like: residual_step with experts' rows", phase, lambda: hy.residual_step(x, None, d, 1e-5, sub=plain, x_in=x, w_next=w, h=h), M * d * (12 + 2 * top))
        del eu, ed, ea, eg, sw, yp, xp, cache, qkvg, q, ao, P
        torch.cuda.empty_cache()
    return bench.rows


def gaparax_kernel_rows(width: int = 4096, prefill: int = 8192, decode: int = 256, ctx: int = 2048, chunk: int = 1024, streams: tuple[int, ...] = (2, 4),
                        experts: int = 64, top: int = 8, expert_ff: int = 1024, dense_ff: int = 16384, softcap: float = 30.0, reach: int = 256) -> list[dict]:
    """The kernels of Gaparax layers, each beside the like kernel of another design ("like: ...")."""
    from ..models.hybrid import distance_buckets
    from ..ops import attention as attn_ops
    from ..ops import hybrid as hy
    from ..ops import moe, paged
    from ..ops.gemm import gemm_tn

    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    bench = _Rows()
    add = bench.add
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dt=bf, sc=1.0: (torch.randn(*s, device=dev, generator=g) * sc).to(dt)      # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)      # noqa: E731
    d, H, hd, bs = width, width // 128, 128, 16
    Hkv, G = H // 4, 4
    table = hy.distance_table(rnd(32, H, dt=f32), distance_buckets(32, reach, chunk), rnd(H, dt=f32) - 4.0)
    for phase, M in (("decode", decode), ("prefill", prefill)):
        one = phase == "decode"
        n_seqs = M if one else M // 2048
        row_seq = i32(list(range(M)) if one else [i // 2048 for i in range(M)])
        c_len = i32([ctx] * n_seqs)
        pos = i32([ctx - 1] * M if one else [i % 2048 for i in range(M)])
        # boundaries of streams: the copies read and written, the result, its gate, the next operand
        w, h, y, gl = rnd(d, dt=f32), rnd(M, d), rnd(M, d), rnd(M, d)
        for n in streams:
            x, coef = rnd(M, n * d, dt=f32), rnd((n + 2) * n, dt=f32, sc=0.3)
            sub = hy.Sublayer(hy.as_out(y), col_gate=hy.as_out(gl), col_bias=w)
            add(f"stream_step, {n} streams, gate", phase, lambda: hy.residual_step(x, None, d, 1e-5, sub=sub, x_in=x, w_next=w, h=h, streams=hy.Streams(n, n, coef)),
                M * d * (6 + 8 * n))
        x = rnd(M, d, dt=f32)
        add("residual_step with gate", phase, lambda: hy.residual_step(x, None, d, 1e-5, sub=sub, x_in=x, w_next=w, h=h), M * d * 14)
        add("like: residual_step (pre-norm frame)", phase, lambda: hy.residual_step(x, None, d, 1e-5, y=hy.as_out(y), x_in=x, w_next=w, h=h), M * d * 12)
        # sigmoid attention in chunks
        ld = Hkv * 2 * hd
        nb = n_seqs * (ctx // bs)
        cache = rnd(nb, bs, ld)
        bt = torch.randperm(nb, device=dev, generator=g).to(torch.int32).view(n_seqs, ctx // bs)
        n = (H + 2 * Hkv) * hd
        P32, wn, temp = rnd(M, n + H * hd, dt=f32), rnd(n, dt=f32), torch.rand(H, device=dev) + 0.5
        P = P32.to(bf)
        q, slot = torch.empty(M, H * hd, dtype=bf, device=dev), i32([i % (nb * bs) for i in range(M)])
        add("gqa_finish_norm, norm of each head", phase, lambda: hy.gqa_finish_norm(hy.as_out(P), None, slot, cache, q, H, Hkv, hd, hd, hd, wn[:hd], wn[:hd], 1e-5, None,
                                                                                   pos, per_head=True, q_scale=temp), M * n * 4)
        if one:
            cols = torch.empty(M, H * hd, dtype=bf, device=dev)
            add("gqa_finish_norm, norm of each head, workspace and gates", phase, lambda: hy.gqa_finish_norm(
                hy.Out(P32, hy.KIND_TAKE), None, slot, cache, q, H, Hkv, hd, hd, hd, wn[:hd], wn[:hd], 1e-5, None, pos, None, True, temp, cols, hd), M * (n + H * hd) * 10)
        freq = torch.tensor([5e5 ** (-2 * i / hd) for i in range(hd // 2)], dtype=torch.float64, device=dev)
        add("like: gqa_finish_norm, norm of all heads, rotation", phase, lambda: hy.gqa_finish_norm(hy.as_out(P), None, slot, cache, q, H, Hkv, hd, hd, hd, wn, wn, 1e-5,
                                                                                                    hy.Rotation(hd, freq), pos), M * n * 4)
        ao, kw = torch.empty(M, H * hd, dtype=bf, device=dev), hy.KeyWeights(table, cols=P[:, n:], pitch=hd)
        if one:
            keys = (ctx - 1) % chunk + 1
            sp = hy.gqa_decode_splits(M, Hkv, chunk)
            args = (q, cache, bt, row_seq, pos, c_len, 0, chunk, hd ** -0.5, 1.0, ao, M, H, Hkv, hd, hd, hd, sp)
            b_, f_ = M * keys * ld * 2 + M * H * hd * 4, 4.0 * M * H * keys * hd
            add(f"gqa_decode chunk {chunk}, sigmoid weights, gates", phase, lambda: hy.gqa_decode(*args, softcap=softcap, weights=kw), b_ + M * H * hd * 2, f_)
            add("like: gqa_decode, softmax, capped", phase, lambda: hy.gqa_decode(*args, softcap=softcap), b_, f_)
            kc, vc = rnd(n_seqs * chunk // bs, bs, Hkv, hd), rnd(n_seqs * chunk // bs, bs, Hkv, hd)
            btd = torch.arange(n_seqs * chunk // bs, dtype=torch.int32, device=dev).view(n_seqs, -1)
            cd = i32([chunk] * M)
            add(f"like: paged_decode ctx {chunk}", phase, lambda: paged.paged_decode(q, kc, vc, btd, cd, H, Hkv, hd, ao), b_, f_)
            del kc, vc
        else:
            plan = hy.plan_prefill([(i, 0, 2048) for i in range(n_seqs)], 0, dev, chunk)
            k, vt = hy.gqa_gather(cache, bt, plan, Hkv, hd, hd)
            pairs = n_seqs * sum(i % chunk + 1 for i in range(2048))
            b_, f_ = (q.numel() + k.numel() + vt.numel() + ao.numel()) * 2, 4.0 * H * pairs * hd
            args = (q, k, vt, k, plan, 0, hd ** -0.5, ao, H, hd, hd, 0, 0, hd)
            add(f"latent_prefill_tc chunk {chunk}, sigmoid weights, gates", phase, lambda: hy.latent_prefill_tc(*args, chunk=chunk, G=G, softcap=softcap, weights=kw),
                b_ + M * H * hd * 2, f_)
            add("the same, not capped", phase, lambda: hy.latent_prefill_tc(*args, chunk=chunk, G=G, weights=kw), b_ + M * H * hd * 2, f_)
            add("like: latent_prefill_tc, softmax, capped", phase, lambda: hy.latent_prefill_tc(*args, chunk=chunk, G=G, softcap=softcap), b_, f_)
            add("like: latent_prefill_tc, softmax", phase, lambda: hy.latent_prefill_tc(*args, chunk=chunk, G=G), b_, f_)
            c = hy.latent_gather(cache, bt, plan)
            args = (q, c, c, plan, 0, hd ** -0.5, ao, H, hd, hd, 0, 0, hd)
            add(f"latent_prefill (any sizes) chunk {chunk}, sigmoid weights, gates", phase, lambda: hy.latent_prefill(*args, chunk=chunk, G=G, softcap=softcap, weights=kw),
                b_ + M * H * hd * 2, f_)
            add("like: latent_prefill (any sizes), softmax, capped", phase, lambda: hy.latent_prefill(*args, chunk=chunk, G=G, softcap=softcap), b_, f_)
            ids = torch.arange(M // chunk, dtype=torch.int32, device=dev).repeat_interleave(chunk)
            ap = attn_ops.make_plan(ids, ids, M, "native")
            qkv = P[:, :n].contiguous()
            add(f"like: tree attention fwd, causal, {chunk} tokens", phase, lambda: attn_ops.forward(qkv, H, Hkv, hd, ap, need_grad=False), b_, f_)
            del qkv, k, vt, c
        del P, P32, cache
        # latent attention without a window, with a sink: d / 128 heads of 128 + 64, latent 512, values 128
        dk, rot, rank, dv = 128, 64, 512, 128
        cache = rnd(nb, bs, rank + rot)
        pq, cn, none = rnd(M, H * (dk + rot) + rank + rot), rnd(rank, dt=f32), i32([-1] * M)
        qn, qr = torch.zeros(H, hy.pad(M, 128), dk, dtype=bf, device=dev), torch.zeros(H, hy.pad(M, 128), rot, dtype=bf, device=dev)
        qe = torch.zeros(M, H * (dk + rot), dtype=bf, device=dev)
        turn = torch.tensor([5e5 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=dev)
        for nxt in (False, True):
            add("like: latent_finish, neighbours" if nxt else "latent_finish, halves", phase, lambda: hy.latent_finish(
                hy.as_out(pq), cn, hy.Rotation(rot, turn, 1.1, nxt), pos, none, cache, M if one else 0, qn, qr, qe, H, dk, rank, 1e-5), M * (2 * H * (dk + rot) + rank + rot) * 2)
        sink = rnd(H, dt=f32)
        if one:
            ql, ol = rnd(H, hy.pad(M, 128), rank), torch.zeros(H, hy.pad(M, 128), rank, dtype=bf, device=dev)
            sp = hy.latent_decode_splits(M, H, ctx)
            for s_ in (sink, None):
                add(f"latent_decode ctx {ctx}, sink" if s_ is not None else "like: latent_decode without sink", phase, lambda: hy.latent_decode(
                    ql, qr, cache, bt, row_seq, pos, c_len, 0, 0.07, ol, M, sp, sink=s_), M * ctx * (rank + rot) * 2 + M * H * (2 * rank + rot) * 2,
                    2.0 * M * H * ctx * (2 * rank + rot))
        else:
            plan = hy.plan_prefill([(i, 0, 2048) for i in range(n_seqs)], 0, dev)
            c = hy.latent_gather(cache, bt, plan)
            k, vt = rnd(plan.n_keys, H * dk), rnd(H * dv, plan.n_keys)
            pairs = n_seqs * 2048 * 2049 // 2
            for s_ in (sink, None):
                add("latent_prefill_tc causal 2048, sink" if s_ is not None else "like: latent_prefill_tc without sink", phase, lambda: hy.latent_prefill_tc(
                    qe, k, vt, c, plan, 0, 0.07, ao, H, dk, dv, rank, rot, dv, weights=hy.KeyWeights(sink=s_)),
                    (qe.numel() + k.numel() + vt.numel() + ao.numel()) * 2, 2.0 * H * pairs * (dk + rot + dv))
            del k, vt, c
        del cache, pq, qn, qr, qe
        # feed-forwards, the residual gate's rows in their input products
        Wu, z = rnd(dense_ff + d, d, sc=d ** -0.5), torch.empty(M, dense_ff + d, dtype=bf, device=dev)
        wb, wf = (Wu.numel() + M * d + z.numel()) * 2, 2.0 * M * d * (dense_ff + d)
        add("gemm_tn up | gate, squared relu of the first columns", phase, lambda: gemm_tn(h, Wu, out=z, relu2=True, relu2_cols=dense_ff), wb, wf)
        add("like: gemm_tn, same product", phase, lambda: gemm_tn(h, Wu, out=z), wb, wf)
        del Wu, z
        logits = rnd(M, experts + d, dt=f32)[:, :experts]
        add("moe.route, best groups", phase, lambda: moe.route(logits, top, False, groups=8, keep=4, scale=2.5), M * (experts * 4 + top * 8))
        add("like: moe.route by logits", phase, lambda: moe.route(logits, top, True), M * (experts * 4 + top * 8))
        rp = moe.route(logits, top, False, groups=8, keep=4, scale=2.5)
        yp = torch.empty(rp.cap_rows, d, dtype=bf, device=dev).normal_()
        gf = rnd(M, d, dt=f32)
        n = streams[0]
        x2, coef = rnd(M, n * d, dt=f32), rnd((n + 2) * n, dt=f32, sc=0.3)
        sub = hy.Sublayer(rows=yp, pos=rp.pos, weight=rp.topw, col_gate=hy.as_out(gf), col_bias=w)
        add(f"stream_step with experts' rows, {n} streams, gate", phase, lambda: hy.residual_step(x2, None, d, 1e-5, sub=sub, x_in=x2, w_next=w, h=h,
                                                                                                 streams=hy.Streams(n, n, coef)), M * d * (6 + 8 * n + 2 * top))
        plain = hy.Sublayer(hy.as_out(y), rows=yp, pos=rp.pos, weight=rp.topw)
        add("like: residual_step with experts' rows", phase, lambda: hy.residual_step(x, None, d, 1e-5, sub=plain, x_in=x, w_next=w, h=h), M * d * (12 + 2 * top))
        del yp, logits
        torch.cuda.empty_cache()
    return bench.rows


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--models", default="nikelix-1b,nikelix-7b")
    ap.add_argument("--batches", default="1,64,256")
    ap.add_argument("--layers", type=int, default=8, help="layers of each preset to run (0: all)")
    ap.add_argument("--part", default="both", choices=["both", "kernels", "engine"])
    a = ap.parse_args()
    for line in report(a.models.split(","), [int(b) for b in a.batches.split(",")], a.layers, a.part):
        print(json.dumps(line), flush=True)


def report(models: list[str], batches: list[int], layers: int, part: str = "both"):
    from ..ops import _lib

    if part != "engine":
        for design, fn in (("nikelix", kernel_rows), ("naselorn", naselorn_kernel_rows), ("gaborax", gaborax_kernel_rows),
                           ("gaparax", gaparax_kernel_rows)):
            if any(m.startswith(design) for m in models):
                yield from ({"part": "kernel", "design": design, **r} for r in fn())
                torch.cuda.empty_cache()
    if part != "kernels":
        yield from ({"part": "engine", **r} for r in engine_rows(models, batches, layers=layers))
    _lib.check_status()


if __name__ == "__main__":
    main()
