"""Gaborax decoders on the GPU against the plain oracle: each mechanism alone and whole models, in fp32 and bf16, as whole
prompts, token by token, in portions, in mixed batches and through the engine's own generation."""
import asyncio
import json
import math
import os
import subprocess

import pytest
import torch

from . import gaborax_oracle as oracle
from .hybrid_models import aligned_gaborax, capped, gaborax, gated_heads, relu2_moe, small_gaborax, yarn
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


def one(*layers, width=68):
    return gaborax(list(layers), vocab=97, width=width)


LAYERS = {
    "gated": (gated_heads(),), "gated-one": (gated_heads(heads=1, kv_heads=1, dim=2, vdim=3, rot=2),),
    "gated-many": (gated_heads(heads=34, kv_heads=2, dim=24, vdim=40, rot=24, scale=0.2),), "gated-partial": (gated_heads(dim=64, vdim=64, rot=16, scale=0.125),),
    "gated-tiles": (gated_heads(heads=6, kv_heads=3, dim=128, vdim=80, rot=128, base=5e4, scale=0.09),),
    "gated-wide": (gated_heads(heads=2, kv_heads=1, dim=40, vdim=264, rot=30, scale=0.2),), "gated-yarn": (gated_heads(rot=20, scaling=yarn(5.0, 32, 4.0, 0.5)),),
    "gated-negative": (gated_heads(dim=64, vdim=64, rot=64, scale=-0.1),), "capped": (capped(),),
    "capped-one": (capped(heads=1, kv_heads=1, dim=4, vdim=4, rot=2, softcap=0.5),), "capped-plain": (capped(heads=4, kv_heads=1, dim=24, vdim=24, rot=24, scaling=None),),
    "capped-tiles": (capped(heads=4, kv_heads=2, dim=64, vdim=96, rot=64, scale=0.5, softcap=4.0),), "capped-wide": (capped(heads=2, kv_heads=2, dim=136, vdim=260, rot=100),),
    "capped-narrow": (capped(heads=3, kv_heads=1, dim=192, vdim=64, rot=72, scale=0.2, softcap=2.0),),
    "shared": (gated_heads(), gated_heads(heads=6, scale=0.5, kv_from=0), capped(), gated_heads(kv_from=0, base=90.0)),
    "shared-tiles": (capped(heads=4, kv_heads=2, dim=64, vdim=64, rot=64), capped(heads=2, kv_heads=2, dim=64, vdim=64, rot=64, softcap=1.5, kv_from=0, scaling=None)),
    "shared-forms": (gated_heads(dim=64, vdim=64, scale=0.2), gated_heads(dim=64, vdim=64, scale=-0.2, kv_from=0), gated_heads(dim=64, vdim=64, kv_from=0)),
}


@DTYPES
@pytest.mark.parametrize("name", list(LAYERS))
def test_attention_layers_prompts_portions_and_decoding(name, dtype):
    d = one(*LAYERS[name])
    toks = tokens(290 if any(x in name for x in ("tiles", "partial", "narrow", "forms")) else 75, 97, 1)
    want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([300], [1], [40, 1], [2], [17, 2, 33, 3], [len(toks) - 2, 2]):
        check(feed(rep, toks, cuts), want, dtype)
    assert rep.bm.num_free == 64 and rep.state_slots is None


@DTYPES
@pytest.mark.parametrize("which", ["small", "aligned"])
def test_whole_model_every_cut(which, dtype):
    d = small_gaborax() if which == "small" else aligned_gaborax()
    toks = tokens(330 if which == "aligned" else 140, d["vocab"], 2)
    want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([len(toks)], [len(toks) - 40, 1], [2, 64, 3, 16, 5, 31], [128, 17]):
        check_routed(feed(rep, toks, cuts), want, dtype, 1.5)


@DTYPES
def test_residual_stream_after_every_layer(dtype):
    from art_b200.engine.runner import SeqView

    d = small_gaborax()
    toks = tokens(33, d["vocab"], 3)
    ref = []
    oracle.forward(d, model(d)[1], toks, torch.float64, ref)
    run = session(d, dtype).runner
    got = run.layer_outputs([SeqView(toks, 0, [5, 2, 9], -1, 0.0, 0, 0)])
    assert len(got) == len(ref) == len(d["layers"])
    for a, b in zip(got, ref):
        err = ((a.cpu() - b).norm(dim=-1) / b.norm(dim=-1)).sort().values
        assert float(err[-1]) < 1e-5 if dtype == F32 else float(err[int(0.9 * len(err))]) < 2e-2


@DTYPES
def test_unequal_requests_in_mixed_batches_reuse_pages(dtype):
    mixed_session(aligned_gaborax(), dtype, [180, 1, 37, 250, 90, 64, 33, 2], check_routed)


@DTYPES
def test_each_request_of_a_batch_equals_itself_alone(dtype):
    d = one(gated_heads(heads=2, kv_heads=1, dim=64, vdim=64, rot=40), capped(heads=2, kv_heads=1), gated_heads(heads=4, kv_heads=1, dim=64, vdim=64, rot=40, kv_from=0))
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


@pytest.mark.parametrize("form", ["scalar32", "scalar16", "decode", "decode-split", "prefill", "tiles"])
@pytest.mark.parametrize("softcap,gated", [(0.0, True), (30.0, False), (8.0, True)])
def test_far_keys_page_borders_caps_and_gates_of_every_attention_form(form, softcap, gated):
    """A key whose score towers above all others lies at the first position, around page and tile borders, at the query
    itself: the output is that key's value times the head's gate, up to what the cap leaves to the others."""
    from art_b200.ops import hybrid as hy

    H, Hkv, bs, n = 4, 2, 16, 420
    dim, vdim = (64, 48) if form == "tiles" else (32, 24)
    dt = F32 if form == "scalar32" else BF16
    rnd = rand(int(softcap) + gated)
    dvp = (hy.prefill_tc_values(dim, 0, vdim, 1.0) if form == "tiles" else 0) or hy.pad(vdim, 16)
    pages = torch.randperm(40, device=DEV)[:27].to(torch.int32)
    for p in (0, 1, 15, 16, 127, 128, 129, 300, 419):
        for j in sorted({0, 1, max(0, p - 1), p, p // 2, p // 16 * 16, max(0, p // 16 * 16 - 1)} & set(range(p + 1))):
            k, v, q = 0.1 * rnd(n, Hkv, dim), rnd(n, Hkv, vdim), rnd(H, dim)
            q = q / q.norm(dim=-1, keepdim=True)
            k[j] += 40.0 * q.view(Hkv, 2, dim).sum(1)
            k, v, q = k.to(dt), v.to(dt), q.to(dt)
            gate = torch.rand(1, H, device=DEV) + 0.1 if gated else None
            cache = torch.zeros(40, bs, Hkv * (dim + dvp), dtype=dt, device=DEV)
            flat, t = cache.view(-1, cache.shape[2]), torch.arange(n, device=DEV)
            rows = pages.long()[t // bs] * bs + t % bs
            flat[rows, :Hkv * dim] = k.reshape(n, -1)
            flat[rows, Hkv * dim:] = torch.nn.functional.pad(v, (0, dvp - vdim)).reshape(n, -1)
            kk, vv = (x[:p + 1].double().repeat_interleave(2, 1) for x in (k, v))
            s = torch.einsum("hd,jhd->hj", q.double(), kk)
            a = torch.softmax(softcap * torch.tanh(s / softcap) if softcap else s, -1)
            want = 0.5 * torch.einsum("hj,jhd->hd", a, vv)
            want = (want * gate.double().view(H, 1) if gated else want).float()
            bt = pages.view(1, -1).contiguous()
            vp = hy.pad(vdim)
            o = torch.full((1, H * vp), 7.0, dtype=dt, device=DEV)
            qq = q.reshape(1, -1).contiguous()
            rest = dict(softcap=softcap, gate=gate)
            if form in ("prefill", "tiles"):
                plan = hy.plan_prefill([(0, p, 1)], 0, DEV)
                rest.update(G=2, out_scale=0.5)
                if form == "tiles":
                    ck, vt = hy.gqa_gather(cache, bt, plan, Hkv, dim, dvp)
                    hy.latent_prefill_tc(qq, ck, vt, ck, plan, 0, 1.0, o, H, dim, dvp, 0, 0, vdim, **rest)
                else:
                    c = hy.latent_gather(cache, bt, plan)
                    hy.latent_prefill(qq, c, c, plan, 0, 1.0, o, H, dim, dvp, 0, 0, vdim, **rest)
            else:
                args = (qq, cache, bt, i32([0]), i32([p]), i32([p + 1]), 0, 0, 1.0, 0.5, o, 1, H, Hkv, dim, vdim, dvp)
                if form.startswith("scalar"):
                    hy.gqa_attend(*args, **rest)
                else:
                    hy.gqa_decode(*args, splits=3 if form == "decode-split" else 1, **rest)
            err = (o.view(H, vp)[:, :vdim].float() - want).norm() / want.norm()
            assert float(err) < (1e-5 if dt == F32 else 2e-2), (p, j, float(err))
            assert vp == vdim or float(o.view(H, vp)[:, vdim:].abs().max()) == 0.0


@pytest.mark.parametrize("H,Hkv,dim,vdim,scale,softcap", [(4, 2, 48, 40, 0.11, 20.0), (6, 1, 128, 128, 0.11, 40.0), (3, 3, 16, 8, 0.3, 5.0), (4, 1, 64, 96, 0.11, 1.0),
                                                          (8, 2, 128, 72, 2.0, 3.0), (2, 1, 192, 128, 0.05, 0.0)])
def test_prompt_attention_tiles_with_caps_and_gates_against_plain_softmax(H, Hkv, dim, vdim, scale, softcap):
    """Several query tiles, sequences that continue a cached prefix, ragged ends; scores on both sides far beyond the cap."""
    from art_b200.ops import hybrid as hy

    rnd = rand(0)
    tc = hy.prefill_tc_values(dim, 0, vdim, scale)
    dvp, G, bs = tc or hy.pad(vdim, 16), H // Hkv, 16
    portions = [(1, 0, 130), (0, 77, 257), (2, 300, 20), (3, 1, 17)]
    plan = hy.plan_prefill(portions, 0, DEV)
    rows = sum(n for _, _, n in portions)
    bt = torch.randperm(4 * 24, device=DEV).to(torch.int32).view(4, 24)
    cache = torch.zeros(4 * 24, bs, Hkv * (dim + dvp), dtype=BF16, device=DEV)
    kv = cache.view(-1, Hkv * (dim + dvp))
    kv[:, :Hkv * dim] = rnd(kv.shape[0], Hkv * dim).to(BF16)
    kv[:, Hkv * dim:].view(-1, Hkv, dvp)[..., :vdim] = rnd(kv.shape[0], Hkv, vdim).to(BF16)
    q = (rnd(rows, H * dim) * 3.0).to(BF16)
    gates = torch.rand(rows + 5, H, device=DEV)
    vp = hy.pad(vdim)
    outs = []
    rest = dict(G=G, softcap=softcap, gate=gates[5:])
    c = hy.latent_gather(cache, bt, plan)
    outs.append(hy.latent_prefill(q, c, c, plan, 0, scale, torch.zeros(rows, H * vp, dtype=BF16, device=DEV), H, dim, dvp, 0, 0, vdim, **rest))
    if tc:
        k, vt = hy.gqa_gather(cache, bt, plan, Hkv, dim, dvp)
        outs.append(hy.latent_prefill_tc(q, k, vt, k, plan, 0, scale, torch.zeros_like(outs[0]), H, dim, dvp, 0, 0, vdim, **rest))
    r0 = 0
    for s, n0, n in portions:
        pos = torch.arange(n0 + n, device=DEV)
        flat = kv[(bt[s].long()[pos // bs] * bs + pos % bs)].double()
        K, V = flat[:, :Hkv * dim].view(-1, Hkv, dim), flat[:, Hkv * dim:].view(-1, Hkv, dvp)[..., :vdim]
        vis = pos[None] <= pos[n0:, None]
        for h in range(H):
            sc = q[r0:r0 + n, h * dim:(h + 1) * dim].double() @ K[:, h // G].T * scale
            sc = softcap * torch.tanh(sc / softcap) if softcap else sc
            ref = torch.softmax(sc.masked_fill(~vis, float("-inf")), -1) @ V[:, h // G]
            for o in outs:
                got = o[r0:r0 + n, h * vp:h * vp + vdim].double() / gates[5 + r0:5 + r0 + n, h:h + 1]
                assert ((got - ref).norm(dim=-1) / ref.norm(dim=-1)).max().item() < 2e-2
        r0 += n


@DTYPES
@pytest.mark.parametrize("H,Hkv,dim,vdim,rot", [(4, 2, 32, 24, 32), (4, 2, 32, 24, 8), (3, 3, 14, 22, 10), (2, 1, 6, 5, 2), (1, 1, 2, 1, 2), (24, 4, 128, 128, 96), (4, 0, 64, 64, 16),
                                                (5, 0, 20, 12, 12), (6, 2, 16, 16, 0), (100, 4, 256, 64, 256)])
def test_norms_rotation_gates_and_cache_write_behind_the_projection(H, Hkv, dim, vdim, rot, dtype):
    """Both pairings, every kind of input, far positions, rows that are not written, sizes of the vector and the scalar form."""
    from art_b200.ops import hybrid as hy

    rnd = rand(H)
    M, dk, dvp, nq, nk, nv = 7, hy.pad(dim, 16), hy.pad(vdim, 16), H * dim, Hkv * dim, Hkv * vdim
    pos = [0, 1, 15, 16, 1000, 131071, 999999]
    slot = [5, 40, -1, 0, 17, 63, 16]
    z = torch.zeros(M, hy.pad(nq + nk + nv + H), device=DEV)
    z[:, :nq + nk + nv + H] = 2 * rnd(M, nq + nk + nv + H)
    bias, wq, wk = rnd(nq + nk + nv), 1 + 0.3 * rnd(nq), 1 + 0.3 * rnd(max(1, nk))
    freq = torch.tensor([300.0 ** (-2 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
    for nxt in (False, True):
        for kind, gated in ((hy.KIND_F32 if dtype == F32 else hy.KIND_BF16, True), (hy.KIND_TAKE, False), (hy.KIND_TAKE, True)):
            zz = z.to(BF16) if kind == hy.KIND_BF16 else z.clone()
            x = zz.double().cpu()[:, :nq + nk + nv]
            x = x + bias.double().cpu() if not gated else x
            cache = torch.full((4, 16, max(1, Hkv) * (dk + dvp)), 3.0, dtype=dtype, device=DEV)
            q, gate = torch.full((M, H * dk), 9.0, dtype=dtype, device=DEV), torch.zeros(M, H, device=DEV) if gated else None
            r = hy.Rotation(rot, freq.to(DEV), 1.25, nxt) if rot else None
            logits = zz.double().cpu()[:, nq + nk + nv:nq + nk + nv + H]
            hy.gqa_finish_norm(hy.Out(zz, kind), None if gated else bias, i32(slot), cache, q, H, Hkv, dim, vdim, dvp, wq, wk if Hkv else None, 1e-5, r, i32(pos), gate)

            def turned(y, heads):
                y = y.view(M, heads, dim).clone()
                src = y.clone()
                for i in range(rot // 2):
                    a, b = (2 * i, 2 * i + 1) if nxt else (i, i + rot // 2)
                    ang = torch.tensor(pos, dtype=torch.float64) * freq[i]
                    c, s = (1.25 * f(ang)[:, None] for f in (torch.cos, torch.sin))
                    y[..., a], y[..., b] = src[..., a] * c - src[..., b] * s, src[..., b] * c + src[..., a] * s
                return y

            tol = 2e-5 if dtype == F32 else 2e-2
            want = turned(oracle.rms(x[:, :nq], 1e-5) * wq.double().cpu(), H)
            got = q.view(M, H, dk).double().cpu()
            assert torch.allclose(got[..., :dim], want, atol=tol * 3, rtol=tol) and (dk == dim or float(got[..., dim:].abs().max()) == 0.0)
            rows = cache.view(64, -1).double().cpu()
            if Hkv:
                wk_ = turned(oracle.rms(x[:, nq:nq + nk], 1e-5) * wk.double().cpu(), Hkv)
                wv = x[:, nq + nk:].view(M, Hkv, vdim)
                for m, sl in enumerate(slot):
                    if sl >= 0:
                        assert torch.allclose(rows[sl, :Hkv * dk].view(Hkv, dk)[:, :dim], wk_[m], atol=tol * 3, rtol=tol)
                        assert torch.allclose(rows[sl, Hkv * dk:].view(Hkv, dvp)[:, :vdim], wv[m], atol=tol, rtol=tol)
            untouched = [i for i in range(64) if i not in slot or not Hkv]
            assert float((rows[untouched] - 3.0).abs().max()) == 0.0
            if gated:
                assert torch.allclose(gate.double().cpu(), oracle.sigmoid(logits), atol=1e-6)
            if kind == hy.KIND_TAKE:
                assert float(zz[:, :nq + nk + nv + (H if gated else 0)].abs().max()) == 0.0


@DTYPES
@pytest.mark.parametrize("experts,identity,top,ff,shared", [(1, 0, 1, 16, 16), (1, 4, 2, 16, 20), (5, 3, 8, 7, 40), (9, 2, 1, 64, 24), (40, 24, 6, 33, 64), (200, 56, 16, 16, 48), (6, 2, 3, 20, None)])
def test_mixture_of_experts_alone(experts, identity, top, ff, shared, dtype):
    """The feed-forward of a layer against the equations; bf16 rows are compared where the choice of experts is no close call."""
    from art_b200.ops import hybrid as hy

    d = one(gated_heads(mlp=relu2_moe(experts, identity, top, ff, shared)))
    run = session(d, dtype).runner
    w = {k[len("l0.mlp."):]: t for k, t in model(d)[1].items() if k.startswith("l0.mlp.")}
    x = torch.zeros(75, run.dp, device=DEV)
    x[:, :68] = rand(2)(75, 68).to(dtype).float()
    h = x.to(dtype)
    from art_b200.engine.runner import SeqView

    b = run._pack([SeqView(tokens(75, 97), 0, [0, 1, 2, 3, 4], -1, 0.0, 0, 0)])[0]
    out = torch.zeros_like(x)
    hy.residual_step(out, None, 68, 1e-5, sub=run._mlp_moe(run.cfg.layers[0], run.layers[0], x, h, b), x_in=torch.zeros_like(x))
    hh = h[:, :68].double().cpu()
    W = {k: t.double() for k, t in w.items()}
    ref = oracle.moe(hh, W, d["layers"][0]["mlp"])
    z = (torch.softmax(hh @ W["router"].T, -1) + W["correction"]).sort(-1, descending=True).values
    clear = torch.ones(75, dtype=torch.bool) if top == experts + identity else z[:, top - 1] - z[:, top] > 3e-5
    err = ((out[:, :68].cpu().double() - ref).norm(dim=-1) / ref.norm(dim=-1))[clear]
    assert int(clear.sum()) > 40 and float(err.max()) < (1e-5 if dtype == F32 else 2e-2)


def test_router_chooses_by_corrected_scores_and_weighs_without_them():
    from art_b200.ops import moe as ops

    z, corr = rand(5)(33, 71), 0.02 * rand(6)(70)
    z[3, :70] = -200.0                                           # far below zero: scores are a softmax all the same
    z[4, 7] = z[4, 9] = 20.0
    corr[7] = corr[9] = 0.0
    z[5, :70] = torch.where(torch.arange(70, device=DEV) == 60, 90.0, -90.0)      # the chosen ones beside it weigh nothing at all
    corr[60] = -2.0
    for norm in (True, False):
        plan = ops.route(z.clone(), 4, norm, correction=corr, identity=20, gate=True)
        s = torch.softmax(z[:, :70].double(), -1)
        top = (s + corr).sort(dim=-1, descending=True, stable=True).indices[:, :4]
        assert torch.equal(plan.topi.long(), top) and plan.topi[4, :2].tolist() == [7, 9] and 60 not in plan.topi[5].tolist()
        a = s.gather(-1, top)
        assert torch.allclose(plan.topw.double(), a / (a.sum(-1, keepdim=True) + 1e-20) if norm else a, atol=1e-6)
        assert float(plan.topw[5].abs().max()) < 1e-10
        assert torch.allclose(plan.gate.double(), oracle.sigmoid(z[:, 70].double()), atol=1e-6)
        assert torch.equal(plan.pos < 0, plan.topi >= 50) and int(plan.counts.sum()) == int((plan.topi < 50).sum()) and bool((plan.topi >= 50).any())
        for m in range(33):                                      # the places of the others hold their token and weight
            for j in range(4):
                if plan.pos[m, j] >= 0:
                    r = int(plan.pos[m, j])
                    assert int(plan.row_token[r]) == m and float(plan.row_w[r]) == float(plan.topw[m, j]) and int(plan.tile_expert[r // 128]) == int(plan.topi[m, j])
    ws = z.clone()
    taken = ops.route(ws, 4, True, take=True, correction=corr, identity=20, gate=True)
    assert float(ws.abs().max()) == 0.0 and torch.equal(taken.topi.long(), top)


def test_residual_step_with_a_row_factor_identity_rows_and_a_plain_copy():
    from art_b200.ops import hybrid as hy

    rnd = rand(1)
    d, dp, M = 101, 104, 6
    for dt in (F32, BF16):
        rows, y, x0, w = (torch.zeros(n, dp, device=DEV) for n in (20, M, M, 1))
        for t in (rows, y, x0, w):
            t[:, :d] = rnd(t.shape[0], d)
        rows = rows.to(dt)
        gate, wk = torch.rand(M, device=DEV), rnd(M, 3)
        pk = torch.randint(-1, 20, (M, 3), device=DEV).int()
        pk[0], pk[1] = -1, i32([3, -1, 4])
        for idn in (x0, x0.to(dt)):
            x, h, ws = x0.clone(), torch.empty(M, dp, dtype=dt, device=DEV), y.clone()
            # the identity rows may be the stream itself, which the step replaces
            sub = hy.Sublayer(hy.Out(ws, hy.KIND_TAKE), rows=rows, pos=pk, weight=wk, gate=gate, identity=hy.as_out(x if idn is x0 else idn))
            hy.residual_step(x, w[0], d, 1e-5, sub=sub, x_in=x, h=h)
            e = torch.where((pk >= 0).unsqueeze(-1), rows.double()[pk.clamp(min=0).long()], idn.double().unsqueeze(1))
            s = gate.double()[:, None] * y.double() + (wk.double().unsqueeze(-1) * e).sum(1)
            want = x0.double()
            want[:, :d] += oracle.rms(s[:, :d], 1e-5) * w[0, :d].double()
            assert torch.allclose(x.double(), want, atol=2e-5) and float(ws.abs().max()) == 0.0
            assert torch.equal(h, x.to(dt))


@pytest.mark.parametrize("M,N,pairs", [(40, 136, False), (300, 264, False), (1030, 520, True)])
def test_squared_relu_in_the_product_epilogue_and_alone(M, N, pairs):
    from art_b200.ops import hybrid as hy
    from art_b200.ops.gemm import gemm_tn

    rnd = rand(N)
    a, W = rnd(M, 128).to(BF16), rnd(N, 128).mul(0.2).to(BF16)
    ref = oracle.relu2(a.double() @ W.double().T)
    assert torch.allclose(gemm_tn(a, W, relu2=True, two_cta=pairs).double(), ref, atol=1e-2, rtol=1e-2)
    z = a.float() @ W.float().T
    for act, f in (("relu2", oracle.relu2), ("relu", lambda t: t.clamp(min=0)), ("silu", lambda t: t * oracle.sigmoid(t))):
        for dt, kind, tol in ((F32, hy.KIND_F32, 1e-5), (F32, hy.KIND_TAKE, 1e-5), (BF16, hy.KIND_TAKE, 1e-2), (BF16, hy.KIND_BF16, 1e-2)):
            zz, out = z.to(BF16) if kind == hy.KIND_BF16 else z.clone(), torch.empty(M, N, dtype=dt, device=DEV)
            hy.plain_act(hy.Out(zz, kind), out, act)
            assert torch.allclose(out.double(), f(zz.double() if kind == hy.KIND_BF16 else z.double()), atol=tol, rtol=tol)
            assert kind != hy.KIND_TAKE or float(zz.abs().max()) == 0.0


def test_squared_relu_in_the_grouped_product():
    from art_b200.ops import moe as ops

    rnd = rand(3)
    E, K, N = 5, 72, 48
    plan = ops.route(rnd(200, E), 2, True)
    x, W = rnd(200, K).to(BF16), rnd(E * N, K).mul(0.2).to(BF16)
    out = ops.grouped_gemm(ops.gather(x, plan), W, plan, N, relu2=True)
    for m in range(0, 200, 7):
        for j in range(2):
            e = int(plan.topi[m, j])
            ref = oracle.relu2(W[e * N:(e + 1) * N].double() @ x[m].double())
            assert torch.allclose(out[int(plan.pos[m, j])].double(), ref, atol=1e-2, rtol=1e-2)


@DTYPES
def test_greedy_generation_through_the_engine(dtype):
    """More requests than the batch holds, prompts in portions beside decoding, shared prefixes from the block cache,
    multi-step decoding with captured graphs; fp32 must reproduce the oracle's greedy tokens, bf16 (no feed-forwards: no close
    calls of a router) its log-probabilities."""
    from art_b200.engine.engine import SamplingParams
    from art_b200.engine.factory import build_engine
    from art_b200.models.config import config_from_dict

    d = small_gaborax()
    if dtype == BF16:
        for e in d["layers"]:
            e["mlp"] = None
    w = model(d, 5)[1]
    eng = build_engine(config_from_dict(d), w, num_blocks=40, max_num_seqs=3, dtype=dtype, max_num_batched_tokens=48, num_scheduler_steps=4)
    common = tokens(37, d["vocab"], 19)
    prompts = [tokens(n, d["vocab"], 20 + n) for n in (5, 61, 30, 1, 118, 17)] + [common + tokens(n, d["vocab"], n) for n in (9, 20)]
    p = SamplingParams(max_tokens=26, temperature=0.0)
    for _ in range(2):                       # the second round replays graphs and reuses pages
        seqs = [eng.add_request(x, p) for x in prompts]
        for _ in range(2000):
            if all(s.finished for s in seqs):
                break
            eng.step()
        eng.step()
        assert all(s.finished for s in seqs) and eng.bm.num_free == 40 and eng.state_slots is None
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
    assert len(eng.runner._dgraphs) >= 1 and eng.bm.stats()["prefix_hits"] > 0
    got = asyncio.run(eng.score(prompts[1], seqs[1].output_ids[:6]))
    assert all(abs(a - b) < (1e-3 if dtype == F32 else 0.1) for a, b in zip(got, seqs[1].logprobs[:6])) and eng.bm.num_free == 40
    sampled = eng.generate_sync(prompts[0], SamplingParams(max_tokens=8, temperature=0.9, top_k=5, top_logprobs=3, seed=1))
    assert len(sampled.output_ids) == 8 and all(len(t) == 3 for t in sampled.top_logprobs)
    eng.runner.close()


@DTYPES
def test_long_decoding_passes_over_pages(dtype):
    d = gaborax([gated_heads(heads=2, kv_heads=1), capped(mlp=relu2_moe(2, 2, 4)), gated_heads(heads=2, kv_heads=1, kv_from=0)], vocab=61, width=64)
    toks = tokens(260, 61, 8)
    check(feed(session(d, dtype), toks, [9, 1]), want_logits(d, toks), dtype, 1.5)


@DTYPES
def test_batched_decoding_with_split_products_and_workspaces(dtype):
    """Wide enough that decode products are split and taken by the kernels behind them; several sequences, every step a
    single token each, against each prompt alone."""
    moe = relu2_moe(5, 1, 6, 64, 256)
    d = gaborax([gated_heads(heads=4, kv_heads=2, dim=64, vdim=64, rot=64, scale=0.125, mlp=moe), capped(heads=8, kv_heads=2, dim=32, vdim=64, rot=32, mlp=moe),
                 gated_heads(heads=4, kv_heads=2, dim=64, vdim=64, rot=64, scale=0.2, kv_from=0)], vocab=304, width=512)
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

    d = small_gaborax()
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
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"],
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

    cfg = resolve_config("gaborax-tiny")
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
