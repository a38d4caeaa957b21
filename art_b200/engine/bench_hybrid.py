"""Throughput of hybrid decoders beside the closest Hugging Face family at equal size (``bench.py --hybrid``).

Two parts, random weights throughout:

* ``engine_rows``: prefill and decode tokens/s of whole models through :class:`~art_b200.engine.engine.Engine`, a hybrid
  preset and a dense Llama-style model of the same width, depth and parameter count per layer, no adapters.
* ``kernel_rows``: every kernel of the hybrid path at the layer sizes of a model, timed alone with CUDA events (L2 flushed
  between calls), with its algorithmic bytes and FLOPs and the fraction of its roofline (the slower of bytes at the
  measured copy bandwidth and FLOPs at the measured tensor or nominal fp32 rate), and the like kernels of the dense model.
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


def dense_twin(cfg):
    """A Llama-style dense model of the same width and depth whose feed-forward (three matrices) has the hybrid's
    parameters (two matrices)."""
    from ..models.config import ModelConfig

    d, ff = cfg.hidden_size, max(s.ff for s in cfg.layers)
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
            for c in (cfg, dense_twin(cfg)):
                r = measure_decode(c, "cuda", seqs=seqs, prompt_len=prompt_len, new_tokens=new_tokens, loras=0)
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


def kernel_rows(width: int = 4096, ff: int = 16384, prefill: int = 8192, decode: int = 256, window: int = 1024, ctx: int = 2048,
                hist: int = 16) -> list[dict]:
    from ..ops import attention as attn_ops
    from ..ops import elementwise as ew
    from ..ops import hybrid as hy
    from ..ops import paged
    from ..ops.gemm import gemm_tn

    dev, bf = "cuda", torch.bfloat16
    gbs, tf = peaks()
    flush = torch.empty(64 << 20, dtype=torch.float32, device=dev)
    rows: list[dict] = []
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dt=bf, sc=1.0: (torch.randn(*s, device=dev, generator=g) * sc).to(dt)      # noqa: E731
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)      # noqa: E731

    def add(name: str, phase: str, fn, bytes_: float, tc_flops: float = 0.0, f32_flops: float = 0.0) -> None:
        us = _time(fn, flush)
        floor = max(bytes_ / gbs / 1e3, tc_flops / tf / 1e6, f32_flops / FP32_TFLOPS / 1e6)
        rows.append({"kernel": name, "phase": phase, "us": round(us, 1), "floor_us": round(floor, 1), "of_roofline": round(floor / us, 3),
                     "gb_s": round(bytes_ / us / 1e3, 0), "tflop_s": round((tc_flops + f32_flops) / us / 1e6, 1)})

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
        inv = rnd(rot // 2, dt=torch.float32)
        cn = rnd(rank, dt=torch.float32)
        slot = i32([-1] * M)
        qn, qr = torch.zeros(H, hy.pad(M, 128), dk, dtype=bf, device=dev), torch.zeros(H, hy.pad(M, 128), rot, dtype=bf, device=dev)
        qe = torch.zeros(M, H * (dk + rot), dtype=bf, device=dev)
        add("latent_finish", phase, lambda: hy.latent_finish(hy.as_out(pq), cn, inv, pos, slot, cache, M if one else 0, qn, qr, qe, H, dk, rot, rank, 1e-5),
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
        yield from ({"part": "kernel", **r} for r in kernel_rows())
        torch.cuda.empty_cache()
    if part != "kernels":
        yield from ({"part": "engine", **r} for r in engine_rows(models, batches, layers=layers))
    _lib.check_status()


if __name__ == "__main__":
    main()
