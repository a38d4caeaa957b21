"""Naselorn decoders on the GPU against the plain oracle: each mechanism alone and whole models, in fp32 and bf16, as whole
prompts, token by token, in portions, in mixed batches and through the engine's own generation."""
import json
import math
import os
import subprocess

import pytest
import torch

from . import naselorn_oracle as oracle
from .hybrid_models import aligned_naselorn, dense, lightning, moe, naselorn, parallel, small_naselorn
from .hybrid_session import BF16, DEV, F32, check, check_routed, feed, mixed_session, model, session, tokens, want_logits

pytestmark = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16])


@pytest.fixture(autouse=True)
def _status_clean():
    yield
    from art_b200.ops import _lib

    torch.cuda.synchronize()
    _lib.check_status()


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def rand(seed):
    g = torch.Generator(device=DEV).manual_seed(seed)
    return lambda *s: torch.randn(*s, device=DEV, generator=g)


def one(layer, width=68):
    return naselorn([layer], vocab=97, width=width)


LAYERS = {
    "lightning": lightning(mlp=dense()), "lightning-tiles": lightning(heads=2, dim=40, vdim=72), "lightning-one": lightning(heads=1, dim=1, vdim=3, decay=[0.5]),
    "lightning-wide": lightning(heads=2, dim=136, vdim=96), "lightning-constant": lightning(heads=3, dim=16, vdim=8, decay=[1.0, 0.9999, 0.05]),
    "parallel": parallel(mlp=dense(33)), "parallel-one": parallel(heads=1, kv_heads=1, dim=4, vdim=4, chunk=1, width=4, blocks=4, conv=1),
    "parallel-many": parallel(heads=34, kv_heads=2, dim=24, vdim=40, chunk=48, width=24, blocks=2, conv=2),
    "parallel-tiles": parallel(heads=6, kv_heads=3, dim=64, vdim=80, chunk=130, width=64, blocks=1, conv=4),
    "parallel-narrow": parallel(heads=3, kv_heads=1, dim=128, vdim=32, chunk=64, width=80, blocks=5, conv=6, left=-0.5, right=2.0),
    "parallel-large": parallel(heads=2, kv_heads=1, dim=96, vdim=264, chunk=37, width=33, blocks=11, conv=3),
    "parallel-long-chunk": parallel(heads=2, kv_heads=2, dim=16, vdim=16, chunk=4096, width=16, blocks=2),
}


@DTYPES
@pytest.mark.parametrize("name", list(LAYERS))
def test_one_layer_prompts_portions_and_decoding(name, dtype):
    d = one(LAYERS[name])
    toks = tokens(290 if "tiles" in name or "narrow" in name else 75, 97, 1)
    want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([300], [1], [40, 1], [2], [17, 2, 33, 3], [len(toks) - 2, 2]):
        check(feed(rep, toks, cuts), want, dtype)
    assert rep.bm.num_free == 64 and rep.state_slots.num_free == 4


@DTYPES
@pytest.mark.parametrize("which", ["small", "aligned"])
def test_whole_model_every_cut(which, dtype):
    d = small_naselorn() if which == "small" else aligned_naselorn()
    toks = tokens(330 if which == "aligned" else 140, d["vocab"], 2)
    want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([len(toks)], [len(toks) - 40, 1], [2, 64, 3, 16, 5, 31], [128, 17]):
        check_routed(feed(rep, toks, cuts), want, dtype, 1.5)


@DTYPES
def test_residual_stream_after_every_layer(dtype):
    from art_b200.engine.runner import SeqView

    d = small_naselorn()
    toks = tokens(33, d["vocab"], 3)
    ref = []
    oracle.forward(d, model(d)[1], toks, torch.float64, ref)
    run = session(d, dtype).runner
    got = run.layer_outputs([SeqView(toks, 0, [5, 2, 9], -1, 0.0, 0, 0, state_slot=3)])
    assert len(got) == len(ref) == len(d["layers"])
    for a, b in zip(got, ref):
        err = ((a.cpu() - b).norm(dim=-1) / b.norm(dim=-1)).sort().values
        assert float(err[-1]) < 1e-5 if dtype == F32 else float(err[int(0.9 * len(err))]) < 2e-2


@DTYPES
def test_unequal_requests_in_mixed_batches_reuse_pages_and_slots(dtype):
    mixed_session(aligned_naselorn(), dtype, [180, 1, 37, 250, 90, 64, 33, 2], check_routed)


@DTYPES
def test_each_request_of_a_batch_equals_itself_alone(dtype):
    d = one(parallel(heads=2, kv_heads=1, dim=64, vdim=64, chunk=40, width=40, blocks=2))
    reqs = {str(i): tokens(n, 97, 50 + i) for i, n in enumerate((130, 1, 61, 18))}
    rep = session(d, dtype)
    cuts = {"0": [97, 2, 31], "1": [1], "2": [3, 1, 57], "3": [1, 17]}
    got = {k: [] for k in reqs}
    for step in range(3):
        entries = []
        for k, c in cuts.items():
            if step < len(c):
                at = sum(c[:step])
                entries.append({"id": k, "tokens": reqs[k][at:at + c[step]], "want": list(range(c[step]))})
        out = rep.step(entries).cpu()
        for e in entries:
            got[e["id"]].append(out[:len(e["tokens"])])
            out = out[len(e["tokens"]):]
    for k, toks in reqs.items():
        check(torch.cat(got[k]), want_logits(d, toks), dtype)


@DTYPES
def test_a_token_is_seen_to_the_end_of_its_chunk_and_by_the_states_at_any_distance(dtype):
    """One changed token shows exactly as far as it must: through the attention branch up to the end of its chunk (chunks
    counted from position 0, wherever portions are cut), through the recurrent ones at any distance."""
    toks = tokens(90, 97, 6)
    other = list(toks)
    other[20] = (toks[20] + 31) % 97
    attn = dict(heads=2, kv_heads=1, width=20, blocks=2, right=0.0)
    cases = [(parallel(chunk=24, **attn), 23), (parallel(chunk=7, dim=64, vdim=64, **attn), 20), (parallel(chunk=30, **attn), 29),
             (parallel(chunk=64, dim=64, vdim=24, **attn), 63), (parallel(left=0.0), 89), (lightning(heads=1, dim=16, vdim=16, decay=[0.9999]), 89)]
    for layer, last in cases:
        d = one(layer)
        if layer["type"] == "parallel":
            w = {k: t.clone() for k, t in model(d)[1].items()}
            w["l0.mix.right.lam"].fill_(-12.0)        # a memory of tens of thousands of tokens
        else:
            w = None
        for cuts in ([90], [50, 1], [30, 7], [10, 12, 2]):
            rep = session(d, dtype, weights=w)
            diff = (feed(rep, toks, cuts) - feed(rep, other, cuts)).abs().amax(-1)
            seen = (diff > 0).nonzero().flatten().tolist()
            assert seen[0] == 20 and seen[-1] == last, (layer["mixer"], cuts, seen[-1])


@pytest.mark.parametrize("form", ["scalar32", "scalar16", "decode", "decode-split", "prefill", "tiles"])
@pytest.mark.parametrize("window,chunk", [(0, 1), (0, 16), (0, 50), (0, 64), (0, 129), (30, 64), (33, 0), (0, 0)])
def test_mask_edges_and_page_borders_of_every_attention_form(form, window, chunk):
    """A key whose score towers above all others is the first one a query sees, then the last one it does not see; the
    query's output must be that key's value, then must not contain it.  Pages are shuffled, positions lie around page borders."""
    from art_b200.ops import hybrid as hy

    H, Hkv, bs, n = 4, 2, 16, 200
    dim, vdim = (64, 48) if form == "tiles" else (32, 24)
    dt = F32 if form == "scalar32" else BF16
    rnd = rand(window + chunk)
    dvp = (hy.prefill_tc_values(dim, 0, vdim, 1.0) if form == "tiles" else 0) or hy.pad(vdim, 16)
    pages = torch.randperm(20, device=DEV)[:13].to(torch.int32)
    for p in (0, 15, 16, 17, 49, 50, 63, 64, 127, 128, 129, 150, 199):
        lo = hy.first_key(p, window, chunk)
        for j in (lo, lo - 1, p):
            if j < 0:
                continue
            k, v, q = 0.1 * rnd(n, Hkv, dim), rnd(n, Hkv, vdim), rnd(H, dim)
            q = q / q.norm(dim=-1, keepdim=True)
            k[j] += 40.0 * q.view(Hkv, 2, dim).sum(1)
            k, v, q = k.to(dt), v.to(dt), q.to(dt)
            cache = torch.zeros(20, bs, Hkv * (dim + dvp), dtype=dt, device=DEV)
            for t in range(n):
                row = cache[pages[t // bs], t % bs]
                row[:Hkv * dim] = k[t].reshape(-1)
                row[Hkv * dim:].view(Hkv, dvp)[:, :vdim] = v[t]
            kk, vv = (x[lo:p + 1].double().repeat_interleave(2, 1) for x in (k, v))
            a = torch.softmax(torch.einsum("hd,jhd->hj", q.double(), kk), -1)
            want = 0.5 * torch.einsum("hj,jhd->hd", a, vv).float()
            bt = pages.view(1, -1).contiguous()
            vp = hy.pad(vdim)
            o = torch.full((1, H * vp), 7.0, dtype=dt, device=DEV)
            qq = q.reshape(1, -1).contiguous()
            if form in ("prefill", "tiles"):
                plan = hy.plan_prefill([(0, p, 1)], window, DEV, chunk)
                rest = dict(chunk=chunk, G=2, out_scale=0.5)
                if form == "tiles":
                    ck, vt = hy.gqa_gather(cache, bt, plan, Hkv, dim, dvp)
                    hy.latent_prefill_tc(qq, ck, vt, ck, plan, window, 1.0, o, H, dim, dvp, 0, 0, vdim, **rest)
                else:
                    c = hy.latent_gather(cache, bt, plan)
                    hy.latent_prefill(qq, c, c, plan, window, 1.0, o, H, dim, dvp, 0, 0, vdim, **rest)
            else:
                args = (qq, cache, bt, i32([0]), i32([p]), i32([p + 1]), window, chunk, 1.0, 0.5, o, 1, H, Hkv, dim, vdim, dvp)
                if form.startswith("scalar"):
                    hy.gqa_attend(*args)
                else:
                    hy.gqa_decode(*args, splits=3 if form == "decode-split" else 1)
            err = (o.view(H, vp)[:, :vdim].float() - want).norm() / want.norm()
            assert float(err) < (1e-5 if dt == F32 else 2e-2), (p, j, float(err))
            assert vp == vdim or float(o.view(H, vp)[:, vdim:].abs().max()) == 0.0


@pytest.mark.parametrize("H,Hkv,dim,vdim,chunk,window", [(4, 2, 48, 40, 100, 0), (6, 1, 128, 128, 300, 0), (3, 3, 16, 8, 7, 0), (4, 1, 64, 96, 0, 0), (2, 2, 64, 64, 129, 0),
                                                         (8, 2, 128, 72, 64, 0), (2, 1, 192, 128, 1, 0), (4, 4, 64, 128, 128, 90)])
def test_prompt_attention_tiles_against_plain_softmax(H, Hkv, dim, vdim, chunk, window):
    """Several query tiles, sequences that continue a cached prefix, ragged ends; strongly negative scores behind tiles of
    which a row sees nothing."""
    from art_b200.ops import hybrid as hy

    rnd = rand(0)
    tc = hy.prefill_tc_values(dim, 0, vdim, 0.11)
    dvp, G, bs = tc or hy.pad(vdim, 16), H // Hkv, 16
    portions = [(1, 0, 130), (0, 77, 257), (2, 300, 20), (3, 1, 17)]
    plan = hy.plan_prefill(portions, window, DEV, chunk)
    rows = sum(n for _, _, n in portions)
    bt = torch.randperm(4 * 24, device=DEV).to(torch.int32).view(4, 24)
    cache = torch.zeros(4 * 24, bs, Hkv * (dim + dvp), dtype=BF16, device=DEV)
    kv = cache.view(-1, Hkv * (dim + dvp))
    kv[:, :Hkv * dim] = (rnd(kv.shape[0], Hkv * dim) - 1.0).to(BF16)
    kv[:, Hkv * dim:].view(-1, Hkv, dvp)[..., :vdim] = rnd(kv.shape[0], Hkv, vdim).to(BF16)
    q = (rnd(rows, H * dim) + 12.0).to(BF16)
    vp = hy.pad(vdim)
    outs = []
    o = torch.zeros(rows, H * vp, dtype=BF16, device=DEV)
    rest = dict(chunk=chunk, G=G)
    if dim % 16 == 0:
        c = hy.latent_gather(cache, bt, plan)
        outs.append(hy.latent_prefill(q, c, c, plan, window, 0.11, o, H, dim, dvp, 0, 0, vdim, **rest))
    if tc:
        k, vt = hy.gqa_gather(cache, bt, plan, Hkv, dim, dvp)
        outs.append(hy.latent_prefill_tc(q, k, vt, k, plan, window, 0.11, torch.zeros_like(o), H, dim, dvp, 0, 0, vdim, **rest))
    r0 = 0
    for s, n0, n in portions:
        pos = torch.arange(n0 + n, device=DEV)
        flat = kv[(bt[s].long()[pos // bs] * bs + pos % bs)].float()
        K, V = flat[:, :Hkv * dim].view(-1, Hkv, dim), flat[:, Hkv * dim:].view(-1, Hkv, dvp)[..., :vdim]
        qpos = pos[n0:]
        vis = pos[None] <= qpos[:, None]
        if chunk:
            vis &= pos[None] // chunk == qpos[:, None] // chunk
        if window:
            vis &= pos[None] > qpos[:, None] - window
        for h in range(H):
            sc = q[r0:r0 + n, h * dim:(h + 1) * dim].float() @ K[:, h // G].T * 0.11
            ref = torch.softmax(sc.masked_fill(~vis, float("-inf")), -1) @ V[:, h // G]
            for o in outs:
                got = o[r0:r0 + n, h * vp:h * vp + vdim].float()
                assert ((got - ref).norm(dim=-1) / ref.norm(dim=-1)).max().item() < 2e-2
        r0 += n


def lightning_reference(q, k, v, decay, S):
    out = []
    for t in range(q.shape[0]):
        S = decay.view(-1, 1, 1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


@pytest.mark.parametrize("n_seqs,H,dim,vdim", [(1, 1, 8, 8), (3, 2, 64, 40), (5, 3, 128, 128), (2, 4, 72, 136), (90, 2, 64, 64), (2, 2, 33, 20), (2, 1, 200, 96)])
def test_lightning_kernels_against_the_recurrence(n_seqs, H, dim, vdim):
    """Chunked tensor-core form, scan and decode: several portion lengths from given states, slow and fast decays, a state
    slot nobody holds, then one token per sequence with a padding row."""
    from art_b200.ops import hybrid as hy

    rnd = rand(dim)
    lens = [(1, 63, 64, 65, 200)[i % 5] if n_seqs < 10 else (i * 7) % 70 + 1 for i in range(n_seqs)]
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    M, nk, nv = cu[-1], H * dim, H * vdim
    p = rnd(M, 2 * nk + nv).to(BF16)
    q, k, v = p[:, :nk], p[:, nk:2 * nk], p[:, 2 * nk:]
    decay = torch.tensor([1 - 0.9 * 0.01 ** h for h in range(H)], device=DEV)
    ld = hy.pad(dim, 4)
    init = torch.zeros(n_seqs + 1, H, vdim, ld, device=DEV)
    init[..., :dim] = rnd(n_seqs + 1, H, vdim, dim)
    slots = list(range(n_seqs, 0, -1))
    fresh = [i % 3 == 1 for i in range(n_seqs)]
    ctx = [n if f else n + 5 for n, f in zip(lens, fresh)]
    silu = lambda t, w: oracle.silu(t.double()).view(-1, H, w)      # noqa: E731
    forms = [("scan", F32, 3e-6), ("scan", BF16, 3e-6)] + ([("tiles", BF16, 2e-5)] if hy.lightning_tc(dim, vdim) else [])
    for form, dt, tol in forms:
        state, o = init.clone(), torch.zeros(M, nv, device=DEV)
        as_ = lambda t: hy.as_out(t.to(dt))      # noqa: E731
        if form == "tiles":
            act = oracle.silu(p.float()).to(BF16)
            hy.lightning_prefill(act[:, :nk], act[:, nk:2 * nk], act[:, 2 * nk:], decay, state, i32(cu), i32(ctx), i32(slots), n_seqs, H, dim, vdim, o)
        else:
            hy.linear_scan(hy.SCAN_FIXED, as_(q), as_(k), as_(v), None, None, decay, state, i32(cu), i32(ctx), i32(slots), n_seqs, H, dim, vdim, o)
        for i in sorted(set(list(range(min(n_seqs, 5))) + [n_seqs - 1])):
            r = slice(cu[i], cu[i + 1])
            qq, kk, vv = silu(q[r], dim), silu(k[r], dim), silu(v[r], vdim)
            S0 = torch.zeros(H, dim, vdim, dtype=torch.float64, device=DEV) if fresh[i] else init[slots[i], ..., :dim].double().transpose(1, 2)
            if form == "tiles":       # with activations that are bf16 numbers the chunked form keeps fp32 accuracy
                qq, kk, vv = (t[r].double().view(-1, H, w) for t, w in ((act[:, :nk], dim), (act[:, nk:2 * nk], dim), (act[:, 2 * nk:], vdim)))
            ref, S = lightning_reference(qq, kk, vv, decay.double(), S0)
            assert ((o[r].view(-1, H, vdim).double() - ref).norm() / ref.norm()).item() < tol
            got = state[slots[i], ..., :dim].transpose(1, 2).double()
            assert ((got - S).norm() / S.norm()).item() < tol
        assert torch.equal(state[0], init[0])
    state = init.clone()
    sl = slots[:-1] + [-1] if n_seqs > 1 else slots
    o = torch.zeros(n_seqs, nv, device=DEV)
    ws = p[:n_seqs].float().contiguous() if M >= n_seqs else None
    P = hy.Out(ws.clone(), hy.KIND_TAKE)
    hy.linear_decode(hy.SCAN_FIXED, P, P.col(nk), P.col(2 * nk), None, None, decay, state, i32(list(range(n_seqs + 1))), i32([9] * n_seqs), i32(sl), H, dim, vdim,
                     None, False, None, o, vdim, 0.0)
    assert float(P.t.abs().max()) == 0.0                       # the workspace is handed back zero
    for i in range(min(n_seqs, 4)):
        if sl[i] < 0:
            continue
        ref, S = lightning_reference(silu(ws[i:i + 1, :nk], dim), silu(ws[i:i + 1, nk:2 * nk], dim), silu(ws[i:i + 1, 2 * nk:], vdim), decay.double(),
                                     init[sl[i], ..., :dim].double().transpose(1, 2))
        assert ((o[i].view(1, H, vdim).double() - ref).norm() / ref.norm()).item() < 3e-6
        assert ((state[sl[i], ..., :dim].transpose(1, 2).double() - S).norm() / S.norm()).item() < 3e-6


@DTYPES
@pytest.mark.parametrize("blocks,bs,taps", [(1, 40, 4), (3, 7, 1), (2, 64, 2), (5, 24, 6)])
def test_convolution_and_gated_recurrence_against_the_equations(blocks, bs, taps, dtype):
    """Portions of several lengths (shorter than the taps, longer than a pass of the scan) from given states, then one
    token per sequence."""
    from art_b200.ops import hybrid as hy

    rnd = rand(bs)
    n, bp, f32 = blocks * bs, hy.pad(bs), dtype == F32
    lens = [700, 1, 2, 3, 256, 17]
    n_seqs = len(lens)
    cu = [0]
    for x in lens:
        cu.append(cu[-1] + x)
    M = cu[-1]
    fresh = [False, True, False, True, True, False]
    ctx = [x if f else x + 9 for x, f in zip(lens, fresh)]
    slots = [3, 0, 5, 2, 6, 1]
    xy = rnd(M, 2 * hy.pad(n)).to(dtype)
    xy[:, n:hy.pad(n)] = 0
    Y, X = hy.as_out(xy), hy.as_out(xy).col(hy.pad(n))
    xb, yb, cb, rb, ib = (0.3 * rnd(n) for _ in range(5))
    conv, lam = rnd(n, taps).to(BF16).float(), 3 * rnd(n) - 3
    ra, ri = (rnd(blocks, bs, bs).mul(bs ** -0.5).to(BF16).float() for _ in range(2))
    decay = 8 * torch.nn.functional.softplus(lam)
    gates = torch.zeros(blocks, 2, bp, bp, device=DEV)
    gates[:, 0, :bs, :bs], gates[:, 1, :bs, :bs] = ra, ri
    gates = gates.view(blocks, 2 * bp, bp)
    gates = gates if f32 else torch.cat([gates, gates], 2).to(BF16)
    state, cst = rnd(7, n), rnd(7, max(1, taps - 1), n)
    s0, c0 = state.clone(), cst.clone()

    def run(Y, X, cu, ctx, slots, M, single):
        ns = len(slots)
        u = torch.zeros(blocks, hy.pad(M, 128), gates.shape[2], dtype=dtype, device=DEV)
        rows = i32([s for s in range(ns) for _ in range(cu[s], cu[s + 1])])
        hy.short_conv(X, xb, conv, cb, cst, rows, i32(cu), i32(ctx), i32(slots), ns, single, u, bs, bp)
        z = torch.empty(M, blocks * 2 * bp, device=DEV)
        hy.gemm_batched(u, gates, z, M, c_batch=2 * bp)
        o = torch.zeros(M, hy.pad(n), dtype=dtype, device=DEV)
        hy.rglru(u, z, rb, ib, decay, Y, yb, state, i32(cu), i32(ctx), i32(slots), ns, single, o, 0.7, bs, bp)
        return o[:, :n]

    def reference(x, y, S, past):
        """x, y [T, n] raw; past [taps - 1, n] inputs before them"""
        full = torch.cat([past, x.double() + xb])
        outs = []
        for t in range(x.shape[0]):
            u = (full[t:t + taps] * conv.double().T).sum(0) + cb
            ub = u.view(blocks, 1, bs)
            r = oracle.sigmoid((ub @ ra.double().transpose(1, 2)).view(-1) + rb)
            i = oracle.sigmoid((ub @ ri.double().transpose(1, 2)).view(-1) + ib)
            a = torch.exp(-8 * r * oracle.softplus(lam.double()))
            S = a * S + torch.sqrt(1 - a * a) * i * u
            outs.append(0.7 * S * oracle.gelu_tanh(y[t].double() + yb))
        return torch.stack(outs), S, full[full.shape[0] - (taps - 1):]

    out = run(Y, X, cu, ctx, slots, M, False)
    tol = 3e-6 if f32 else 4e-3
    zero = torch.zeros(taps - 1, n, dtype=torch.float64, device=DEV)
    for s in range(n_seqs):
        r = slice(cu[s], cu[s + 1])
        past = zero if fresh[s] else c0[slots[s], :taps - 1].double()
        ref, S, tail = reference(X.t[r, :n], xy[r, :n], torch.zeros(n, dtype=torch.float64, device=DEV) if fresh[s] else s0[slots[s]].double(), past)
        assert ((out[r].double() - ref).norm() / ref.norm()).item() < tol
        assert ((state[slots[s]].double() - S).norm() / S.norm()).item() < (3e-6 if f32 else 2e-5)      # the state is fp32 in both
        if taps > 1:
            assert torch.allclose(cst[slots[s], :taps - 1].double(), tail, atol=1e-6)
    assert torch.equal(state[4], s0[4]) and torch.equal(cst[4], c0[4])
    s1, c1 = state.clone(), cst.clone()
    ws = rnd(4, 2 * hy.pad(n))
    take = hy.Out(ws.clone(), hy.KIND_TAKE)
    sl = [6, -1, 2, 0]
    out = run(take, take.col(hy.pad(n)), [0, 1, 2, 3, 4], [5, 0, 1, 8], sl, 4, True)
    assert float(take.t[:, :n].abs().max()) == 0.0 and float(take.t[:, hy.pad(n):hy.pad(n) + n].abs().max()) == 0.0
    for m in (0, 2, 3):
        new = m == 2                                             # its first token: whatever the slot holds is ignored
        ref, S, tail = reference(ws[m:m + 1, hy.pad(n):hy.pad(n) + n], ws[m:m + 1, :n], 0 * s1[sl[m]].double() if new else s1[sl[m]].double(),
                                 zero if new else c1[sl[m], :taps - 1].double())
        assert ((out[m].double() - ref[0]).norm() / ref.norm()).item() < tol
        assert ((state[sl[m]].double() - S).norm() / S.norm()).item() < (3e-6 if f32 else 2e-5)
        if taps > 1:
            assert torch.allclose(cst[sl[m], :taps - 1].double(), tail, atol=1e-6)


@DTYPES
@pytest.mark.parametrize("experts,top,ff,shared", [(1, 1, 16, 16), (5, 5, 7, 40), (9, 1, 64, 24), (40, 6, 33, 64), (200, 16, 16, 48)])
def test_mixture_of_experts_alone(experts, top, ff, shared, dtype):
    """The feed-forward of a layer against the equations; bf16 rows are compared where the choice of experts is no close call."""
    from art_b200.ops import hybrid as hy

    d = one(lightning(mlp=moe(experts, top, ff, shared)))
    run = session(d, dtype).runner
    w = {k[len("l0.mlp."):]: t for k, t in model(d)[1].items() if k.startswith("l0.mlp.")}
    h = torch.zeros(75, run.dp, device=DEV)
    h[:, :68] = rand(2)(75, 68)
    h = h.to(dtype)
    x = torch.zeros(75, run.dp, device=DEV)
    b = run._pack([_view(tokens(75, 97))])[0]
    hy.residual_step(x, None, 68, 1e-5, sub=run._mlp_moe(run.cfg.layers[0], run.layers[0], None, h, b), x_in=torch.zeros_like(x))
    hh = h[:, :68].double().cpu()
    W = {k: t.double() for k, t in w.items()}
    ref = oracle.moe(hh, W, d["layers"][0]["mlp"])
    z = (hh @ W["router"].T + W["router.b"]).sort(-1, descending=True).values
    clear = torch.ones(75, dtype=torch.bool) if top == experts else z[:, top - 1] - z[:, top] > 1e-3
    err = ((x[:, :68].cpu().double() - ref).norm(dim=-1) / ref.norm(dim=-1))[clear]
    assert int(clear.sum()) > 40 and float(err.max()) < (1e-5 if dtype == F32 else 2e-2)


def _view(toks):
    from art_b200.engine.runner import SeqView

    return SeqView(toks, 0, list(range(len(toks) // 16 + 1)), -1, 0.0, 0, 0, state_slot=0)


def test_router_chooses_the_largest_biased_logits_and_breaks_ties_by_index():
    from art_b200.ops import moe as ops

    z, bias = rand(5)(33, 70), rand(6)(70)
    z[3] = -200.0                                                # far below zero: weights stay a softmax over the chosen
    z[4, 7] = z[4, 9] = 50.0
    bias[7] = bias[9] = 0.0
    for norm in (True, False):
        plan = ops.route(z.clone(), 4, norm, bias)
        s = (z + bias).double()
        top = s.sort(dim=-1, descending=True, stable=True).indices[:, :4]
        assert torch.equal(plan.topi.long(), top) and plan.topi[4, :2].tolist() == [7, 9]
        want = torch.softmax(s.gather(-1, top), -1) if norm else torch.softmax(s, -1).gather(-1, top)
        assert torch.allclose(plan.topw.double(), want, atol=1e-6)
    ws = z.clone()
    taken = ops.route(ws, 4, True, bias, take=True)
    assert float(ws.abs().max()) == 0.0 and torch.equal(taken.topi.long(), top)


def test_residual_step_without_a_norm_experts_bias_and_position_vectors():
    from art_b200.ops import hybrid as hy

    rnd = rand(1)
    d, dp, M = 101, 104, 6
    for dt, tol in ((F32, 1e-5), (BF16, 1e-2)):
        table = torch.zeros(11, dp, device=DEV)
        table[:, :d] = rnd(11, d)
        table = table.to(dt)
        pos = [0, 1, 7, 1000, 131071, 999999]
        freq = torch.tensor([10000.0 ** (-2.0 * i / d) for i in range(dp // 2)], dtype=torch.float64, device=DEV)
        x, h, w = torch.empty(M, dp, device=DEV), torch.empty(M, dp, dtype=dt, device=DEV), torch.zeros(dp, device=DEV)
        w[:d] = rnd(d)
        tok = torch.tensor([3, 10, 0, 5, 5, 1], device=DEV)
        hy.residual_step(x, None, d, 1e-5, mult=3.0, tokens=tok, table=table, freq=freq, pos=i32(pos), w_next=w, h=h)
        c = torch.arange(d, dtype=torch.float64)
        ang = torch.tensor(pos, dtype=torch.float64)[:, None] * 10000.0 ** (-2.0 * (c // 2) / d)
        ref = 3.0 * table[tok, :d].double().cpu() + torch.where(c % 2 == 0, torch.sin(ang), torch.cos(ang))
        assert torch.allclose(x[:, :d].double().cpu(), ref, atol=1e-5) and float(x[:, d:].abs().max()) == 0.0
        assert torch.allclose(h[:, :d].double().cpu(), oracle.rms(ref, 1e-5) * w[:d].double().cpu(), atol=3 * tol)
        rows, bias, y = torch.zeros(20, dp, device=DEV), torch.zeros(dp, device=DEV), torch.zeros(M, dp, device=DEV)
        rows[:, :d], bias[:d], y[:, :d] = rnd(20, d), rnd(d), rnd(M, d)
        rows = rows.to(dt)
        pk, wk = torch.randint(0, 20, (M, 3), device=DEV).int(), rnd(M, 3)
        ws = y.clone()
        x0 = x.clone()
        hy.residual_step(x, None, d, 1e-5, sub=hy.Sublayer(hy.Out(ws, hy.KIND_TAKE), bias, rows, pk, wk), x_in=x0)
        want = x0.double() + y.double() + bias.double() + (wk.double().unsqueeze(-1) * rows[pk.long()].double()).sum(1)
        assert torch.allclose(x.double(), want, atol=1e-5) and float(ws.abs().max()) == 0.0


@pytest.mark.parametrize("n", [16, 48, 336, 4096])
def test_gated_activation_and_row_norm(n):
    from art_b200.ops import hybrid as hy

    rnd = rand(n)
    gate, up = rnd(9, n), rnd(9, n)
    z = torch.stack([gate.view(9, -1, 16), up.view(9, -1, 16)], 2).reshape(9, 2 * n)
    for act, f in (("silu", oracle.silu), ("relu", lambda t: t.clamp(min=0))):
        for dt, tol in ((F32, 1e-5), (BF16, 2e-2)):
            for kind in ((hy.KIND_F32, hy.KIND_TAKE) if dt == F32 else (hy.KIND_BF16, hy.KIND_TAKE)):
                zz = z.to(BF16) if kind == hy.KIND_BF16 else z.clone()
                out = torch.empty(9, n, dtype=dt, device=DEV)
                hy.gated_act(hy.Out(zz, kind), out, act)
                assert torch.allclose(out.double(), f(gate.double()) * up.double(), atol=tol * 4)
                assert kind != hy.KIND_TAKE or float(zz.abs().max()) == 0.0
    for m in (n, n - 3):                       # a row of whole vectors and an odd one
        o, w, g = rnd(9, m), rnd(m), rnd(9, m)
        out = torch.full((9, hy.pad(m)), 5.0, device=DEV)
        hy.head_norm(o, w, False, 1, m, hy.pad(m), out, 1e-5, hy.as_out(g), hy.GATE_SIGMOID)
        ref = oracle.rms(o.double(), 1e-5) * w.double() * oracle.sigmoid(g.double())
        assert torch.allclose(out[:, :m].double(), ref, atol=1e-5) and (m == hy.pad(m) or float(out[:, m:].abs().max()) == 0.0)


@pytest.mark.parametrize("M,pairs", [(64, False), (1100, True)])
def test_relu_gate_in_the_product_epilogue(M, pairs):
    from art_b200.ops.gemm import gemm_tn

    rnd = rand(M)
    K, n = 192, 288
    a, wg, wu = rnd(M, K).to(BF16), rnd(n, K).mul(K ** -0.5).to(BF16), rnd(n, K).mul(K ** -0.5).to(BF16)
    W = torch.stack([wg.view(-1, 16, K), wu.view(-1, 16, K)], 1).reshape(2 * n, K).contiguous()
    for act, f in (("relu", lambda t: t.clamp(min=0)), ("silu", oracle.silu)):
        out = torch.empty(M, n, dtype=BF16, device=DEV)
        assert gemm_tn(a, W, swiglu_out=out, gate_act=act, keep_preact=False, two_cta=pairs) is None
        ref = f(a.double() @ wg.double().T) * (a.double() @ wu.double().T)
        assert ((out.double() - ref).norm() / ref.norm()).item() < 1e-2


@pytest.mark.parametrize("M,N,cols,pairs", [(40, 136, 72, False), (300, 264, 264, False), (1030, 520, 392, True)])
def test_silu_of_the_first_columns_in_the_product_epilogue(M, N, cols, pairs):
    from art_b200.ops.gemm import gemm_tn

    rnd = rand(N)
    a, W = rnd(M, 128).to(BF16), rnd(N, 128).mul(0.2).to(BF16)
    out = gemm_tn(a, W, silu_cols=cols, two_cta=pairs)
    ref = a.double() @ W.double().T
    ref[:, :cols] = oracle.silu(ref[:, :cols])
    assert torch.allclose(out.double(), ref, atol=1e-2, rtol=1e-2)


@DTYPES
def test_greedy_generation_through_the_engine(dtype):
    """More requests than state slots, prompts in portions beside decoding, multi-step decoding with captured graphs; fp32
    must reproduce the oracle's greedy tokens, bf16 (dense feed-forwards: no close calls of a router) its log-probabilities."""
    from art_b200.engine.engine import SamplingParams
    from art_b200.engine.factory import build_engine
    from art_b200.models.config import config_from_dict

    d = small_naselorn()
    if dtype == BF16:
        for e in d["layers"]:
            e["mlp"] = dense(44)
    w = model(d, 5)[1]
    eng = build_engine(config_from_dict(d), w, num_blocks=40, max_num_seqs=3, dtype=dtype, max_num_batched_tokens=48, num_scheduler_steps=4)
    prompts = [tokens(n, d["vocab"], 20 + n) for n in (5, 61, 30, 1, 118, 17)]
    p = SamplingParams(max_tokens=26, temperature=0.0)
    for _ in range(2):                       # the second round replays graphs and reuses pages and slots
        seqs = [eng.add_request(x, p) for x in prompts]
        for _ in range(2000):
            if all(s.finished for s in seqs):
                break
            eng.step()
        eng.step()
        assert all(s.finished for s in seqs) and eng.bm.num_free == 40 and eng.state_slots.num_free == 3
        for x, s in zip(prompts, seqs):
            full = oracle.forward(d, w, x + s.output_ids, torch.float64)[len(x) - 1:-1]
            lp = torch.log_softmax(full, -1)
            mine = lp.gather(-1, torch.tensor(s.output_ids).unsqueeze(-1)).squeeze(-1)
            if dtype == F32:
                assert s.output_ids == full.argmax(-1).tolist()
                assert torch.allclose(torch.tensor(s.logprobs, dtype=torch.float64), mine, atol=1e-4)
            else:
                assert float((lp.amax(-1) - mine).max()) < 0.3       # the token taken is the best one or a near-tie
                assert torch.allclose(torch.tensor(s.logprobs, dtype=torch.float64), mine, atol=0.2)
    assert len(eng.runner._dgraphs) >= 1
    sampled = eng.generate_sync(prompts[0], SamplingParams(max_tokens=8, temperature=0.9, top_k=5, top_logprobs=3, seed=1))
    assert len(sampled.output_ids) == 8 and all(len(t) == 3 for t in sampled.top_logprobs)
    eng.runner.close()


@DTYPES
def test_long_decoding_passes_over_chunks_and_pages(dtype):
    d = naselorn([parallel(chunk=40, heads=2, kv_heads=1), lightning(mlp=dense()), parallel(chunk=16, width=20, blocks=2)], vocab=61, width=64)
    toks = tokens(260, 61, 8)
    check(feed(session(d, dtype), toks, [9, 1]), want_logits(d, toks), dtype, 1.5)


@DTYPES
def test_batched_decoding_with_split_products_and_workspaces(dtype):
    """Wide enough that decode products are split and taken by the kernels behind them; several sequences, every step a
    single token each, against each prompt alone."""
    d = naselorn([lightning(heads=4, dim=64, vdim=64, mlp=dense(512)), parallel(heads=4, kv_heads=2, dim=64, vdim=64, chunk=24, width=256, blocks=4, conv=4,
                  mlp=moe(6, 6, 64, 256))], vocab=304, width=512)
    reqs = [tokens(40, 304, 70 + i) for i in range(4)]
    rep = session(d, dtype)
    got = [[] for _ in reqs]
    for t in range(40):
        out = rep.step([{"id": str(i), "tokens": [r[t]], "want": [0]} for i, r in enumerate(reqs)]).cpu()
        for i in range(4):
            got[i].append(out[i:i + 1])
    for g, r in zip(got, reqs):
        check(torch.cat(g), want_logits(d, r), dtype, 1.5)
    if dtype == BF16:
        assert any(k[0] == "ws" for k in rep.runner._buf)


def test_trace_command_line(tmp_path):
    import numpy as np
    from safetensors.torch import save_file

    d = small_naselorn()
    _, w = model(d, 7)
    (tmp_path / "m").mkdir()
    (tmp_path / "m" / "config.json").write_text(json.dumps(d))
    save_file(w, str(tmp_path / "m" / "model.safetensors"))
    toks = tokens(40, d["vocab"], 9)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[31:], "want": [8]}, {"id": "y", "tokens": toks[:3], "want": [2]}], "end": ["x", "y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    ref = oracle.forward(d, w, toks, torch.float64).float()
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=180)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    for step, rows in ((0, [0, 29]), (2, [39, 2])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").copy()).view(len(rows), d["vocab"])
        check(got, ref[rows], F32)


def test_preset_is_served_by_the_engine():
    from art_b200.engine.engine import SamplingParams
    from art_b200.engine.factory import build_engine
    from art_b200.models.config import resolve_config
    from art_b200.models.weights import init_base_weights

    cfg = resolve_config("naselorn-tiny")
    eng = build_engine(cfg, init_base_weights(cfg, dtype=BF16, device=DEV), num_blocks=64, max_num_seqs=4, eos_token_id=None)
    seqs = [eng.add_request(tokens(n, cfg.vocab_size, n), SamplingParams(max_tokens=12, temperature=0.7, seed=n)) for n in (3, 50, 21)]
    for _ in range(200):
        if all(s.finished for s in seqs):
            break
        eng.step()
    assert all(len(s.output_ids) == 12 and all(math.isfinite(x) for x in s.logprobs) for s in seqs)
    with pytest.raises(ValueError, match="adapters"):
        eng.runner.set_adapter(0, {})
    eng.runner.close()
