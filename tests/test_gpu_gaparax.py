"""Gaparax decoders on the GPU against the plain oracle: each mechanism alone and whole models, in fp32 and bf16, as whole
prompts, token by token, in portions, in mixed batches and through the engine's own generation."""
import asyncio
import json
import math
import os
import subprocess

import pytest
import torch

from . import gaparax_oracle as oracle
from .hybrid_models import aligned_gaparax, gaparax, group_moe, relu2_dense, sigmoid_heads, sink_latent, small_gaparax, yarn
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


def one(*layers, width=68, streams=2):
    return gaparax(list(layers), vocab=97, width=width, streams=streams)


LAYERS = {
    "sigmoid": (sigmoid_heads(),), "sigmoid-one": (sigmoid_heads(heads=1, kv_heads=1, dim=2, vdim=3, chunk=5, bias_max=3),),
    "sigmoid-many": (sigmoid_heads(heads=34, kv_heads=2, dim=24, vdim=40, chunk=64, scale=0.2, bias_max=40),),
    "sigmoid-tiles": (sigmoid_heads(heads=6, kv_heads=3, dim=128, vdim=80, chunk=140, scale=0.09, softcap=20.0, bias_max=100),),
    "sigmoid-square": (sigmoid_heads(heads=4, kv_heads=4, dim=64, vdim=64, chunk=129, scale=0.125, bias_max=500),),
    "sigmoid-uncapped": (sigmoid_heads(heads=4, kv_heads=1, dim=64, vdim=72, chunk=300, softcap=None, bias_max=30),),
    "sigmoid-narrow": (sigmoid_heads(heads=3, kv_heads=1, dim=192, vdim=64, chunk=100, scale=0.1, softcap=2.0, bias_max=50),),
    "sigmoid-wide": (sigmoid_heads(heads=2, kv_heads=1, dim=40, vdim=264, chunk=33, bias_max=20),),
    "sigmoid-negative": (sigmoid_heads(dim=64, vdim=64, chunk=31, scale=-0.1, bias_max=8),), "sigmoid-single": (sigmoid_heads(chunk=1, bias_max=2),),
    "sink": (sink_latent(),), "sink-one": (sink_latent(heads=1, dim=2, rot=2, rank=4, vdim=1, scaling=None),),
    "sink-many": (sink_latent(heads=35, dim=24, rot=16, rank=96, vdim=40),), "sink-plain": (sink_latent(rot=24, scaling=None, base=2000.0),),
    "sink-tiles": (sink_latent(heads=3, dim=64, rot=64, rank=100, vdim=56, scale=0.1),),
    "sink-large": (sink_latent(heads=18, dim=128, rot=64, rank=512, vdim=128, scale=0.06, base=5e4, scaling=yarn(4.0, 64, 8.0, 1.0)),),
    "sink-wide": (sink_latent(heads=2, dim=20, rot=8, rank=40, vdim=136),), "sink-deep": (sink_latent(heads=2, dim=16, rot=16, rank=800, vdim=16),),
    "sink-negative": (sink_latent(heads=2, dim=64, rot=64, rank=48, vdim=64, scale=-0.1),),
}


@DTYPES
@pytest.mark.parametrize("name", list(LAYERS))
def test_attention_layers_prompts_portions_and_decoding(name, dtype):
    d = one(*LAYERS[name])
    toks = tokens(290 if any(x in name for x in ("tiles", "square", "narrow", "uncapped")) else 75, 97, 1)
    want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([300], [1], [40, 1], [2], [17, 2, 33, 3], [len(toks) - 2, 2]):
        check(feed(rep, toks, cuts), want, dtype)
    assert rep.bm.num_free == 64 and rep.state_slots is None


@DTYPES
@pytest.mark.parametrize("streams", [1, 2, 4, 7])
def test_hyper_connections_of_several_widths(streams, dtype):
    d = gaparax([sigmoid_heads(mlp=relu2_dense(50)), sink_latent(), sigmoid_heads(heads=2, mlp=relu2_dense(24))], vocab=101, width=76, streams=streams)
    toks = tokens(60, 101, 2)
    for layers in (d["layers"], d["layers"][:1], d["layers"][1:2]):      # the first sublayer may be the last one
        e = {**d, "layers": layers}
        rep = session(e, dtype)
        for cuts in ([60], [1], [19, 2, 30]):
            check(feed(rep, toks, cuts), want_logits(e, toks), dtype)


@DTYPES
@pytest.mark.parametrize("which", ["small", "aligned"])
def test_whole_model_every_cut(which, dtype):
    d = small_gaparax() if which == "small" else aligned_gaparax()
    toks = tokens(330 if which == "aligned" else 140, d["vocab"], 2)
    want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([len(toks)], [len(toks) - 40, 1], [2, 64, 3, 16, 5, 31], [128, 17]):
        check_routed(feed(rep, toks, cuts), want, dtype, 1.5)


@DTYPES
def test_residual_stream_after_every_layer(dtype):
    from art_b200.engine.runner import SeqView

    d = small_gaparax()
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
    mixed_session(aligned_gaparax(), dtype, [180, 1, 37, 250, 90, 64, 33, 2], check_routed)


@DTYPES
def test_each_request_of_a_batch_equals_itself_alone(dtype):
    d = one(sigmoid_heads(heads=2, kv_heads=1, dim=64, vdim=64, chunk=40), sink_latent(heads=2, dim=64, rot=64, vdim=48), sigmoid_heads(chunk=16, mlp=relu2_dense()))
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
@pytest.mark.parametrize("softcap,chunk,pitched", [(0.0, 0, True), (20.0, 100, False), (9.0, 16, True), (15.0, 128, False)])
def test_far_keys_borders_biases_and_gates_of_every_sigmoid_form(form, softcap, chunk, pitched):
    """All keys but one weigh next to nothing; that one lies at the first position, around page, tile and chunk borders, at the
    query itself, just inside and just outside the chunk: the output is its value times its weight and the columns' gate."""
    from art_b200.models.hybrid import distance_buckets
    from art_b200.ops import hybrid as hy

    H, Hkv, bs, n = 4, 2, 16, 420
    dim, vdim = (64, 48) if form == "tiles" else (32, 20)
    dt = F32 if form == "scalar32" else BF16
    rnd = rand(int(softcap) + chunk)
    dvp = (hy.prefill_tc_values(dim, 0, vdim, 1.0) if form == "tiles" else 0) or hy.pad(vdim, 16)
    pages = torch.randperm(40, device=DEV)[:27].to(torch.int32)
    reach = 300
    rel = -5.0 + 0.3 * rnd(28, H)
    pb = 0.2 * rnd(H)
    table = hy.distance_table(rel, distance_buckets(28, reach, chunk), pb)
    for p in (0, 1, 15, 16, 99, 100, 127, 128, 129, 255, 256, 300, 419):
        first = p - p % chunk if chunk else 0
        for j in sorted({0, 1, first, first + 1, first - 1, p, p - 1, (first + p) // 2, p // 16 * 16, p // 16 * 16 - 1} & set(range(p + 1))):
            k, v, q = 0.1 * rnd(n, Hkv, dim), rnd(n, Hkv, vdim), rnd(H, dim)
            q = 8 * q / q.norm(dim=-1, keepdim=True)
            k[j] += q.view(Hkv, 2, dim).sum(1) / 6
            k, v, q = k.to(dt), v.to(dt), q.to(dt)
            cache = torch.zeros(40, bs, Hkv * (dim + dvp), dtype=dt, device=DEV)
            flat, t = cache.view(-1, cache.shape[2]), torch.arange(n, device=DEV)
            rows = pages.long()[t // bs] * bs + t % bs
            flat[rows, :Hkv * dim] = k.reshape(n, -1)
            flat[rows, Hkv * dim:] = torch.nn.functional.pad(v, (0, dvp - vdim)).reshape(n, -1)
            vp = hy.pad(vdim)
            pitch = vp if pitched else vdim
            cols = torch.full((1, H * pitch + 8), float("nan"), dtype=dt, device=DEV)      # what lies between the gates is not used
            z = rnd(1, H, vdim).to(dt)
            cols[:, :H * pitch].view(1, H, pitch)[..., :vdim] = z
            kk, vv = (x[first:p + 1].double().repeat_interleave(2, 1) for x in (k, v))
            s = torch.einsum("hd,jhd->hj", q.double(), kk)
            s = softcap * torch.tanh(s / softcap) if softcap else s
            b = torch.stack([rel.double()[oracle.bucket(p - x, 28, reach)] + pb.double() for x in range(first, p + 1)], 1)
            want = 0.5 * torch.einsum("hj,jhd->hd", oracle.sigmoid(s + b), vv) * oracle.sigmoid(z[0].double())
            bt = pages.view(1, -1).contiguous()
            o = torch.full((1, H * vp), 7.0, dtype=dt, device=DEV)
            qq = q.reshape(1, -1).contiguous()
            rest = dict(softcap=softcap, weights=hy.KeyWeights(table, cols=cols, pitch=pitch))
            if form in ("prefill", "tiles"):
                plan = hy.plan_prefill([(0, p, 1)], 0, DEV, chunk)
                rest.update(G=2, out_scale=0.5, chunk=chunk)
                if form == "tiles":
                    ck, vt = hy.gqa_gather(cache, bt, plan, Hkv, dim, dvp)
                    hy.latent_prefill_tc(qq, ck, vt, ck, plan, 0, 1.0, o, H, dim, dvp, 0, 0, vdim, **rest)
                else:
                    c = hy.latent_gather(cache, bt, plan)
                    hy.latent_prefill(qq, c, c, plan, 0, 1.0, o, H, dim, dvp, 0, 0, vdim, **rest)
            else:
                args = (qq, cache, bt, i32([0]), i32([p]), i32([p + 1]), 0, chunk, 1.0, 0.5, o, 1, H, Hkv, dim, vdim, dvp)
                if form.startswith("scalar"):
                    hy.gqa_attend(*args, **rest)
                else:
                    hy.gqa_decode(*args, splits=3 if form == "decode-split" else 1, **rest)
            err = (o.view(H, vp)[:, :vdim].double() - want).norm() / want.norm()
            assert float(err) < (2e-5 if dt == F32 else 2e-2), (p, j, float(err))
            assert vp == vdim or float(o.view(H, vp)[:, vdim:].abs().max()) == 0.0


@pytest.mark.parametrize("H,Hkv,dim,vdim,scale,softcap,chunk,reach", [(4, 2, 48, 40, 0.11, 20.0, 0, 700), (6, 1, 128, 128, 0.11, 40.0, 150, 64), (3, 3, 16, 8, 0.3, 5.0, 200, 20),
                                                                     (4, 1, 64, 96, 0.11, 1.0, 0, 40), (8, 2, 128, 72, 2.0, 3.0, 64, 300), (2, 1, 192, 128, 0.05, 0.0, 0, 129)])
def test_prompt_attention_with_sigmoid_weights_against_plain_ones(H, Hkv, dim, vdim, scale, softcap, chunk, reach):
    """Several query tiles, sequences that continue a cached prefix, ragged ends; every distance has a bias of its own, so that a
    table that is off by one shows."""
    from art_b200.ops import hybrid as hy

    rnd = rand(0)
    tc = hy.prefill_tc_values(dim, 0, vdim, scale)
    dvp, G, bs = tc or hy.pad(vdim, 16), H // Hkv, 16
    portions = [(1, 0, 130), (0, 77, 257), (2, 300, 20), (3, 1, 17)]
    plan = hy.plan_prefill(portions, 0, DEV, chunk)
    rows = sum(n for _, _, n in portions)
    bt = torch.randperm(4 * 24, device=DEV).to(torch.int32).view(4, 24)
    cache = torch.zeros(4 * 24, bs, Hkv * (dim + dvp), dtype=BF16, device=DEV)
    kv = cache.view(-1, Hkv * (dim + dvp))
    kv[:, :Hkv * dim] = rnd(kv.shape[0], Hkv * dim).to(BF16)
    kv[:, Hkv * dim:].view(-1, Hkv, dvp)[..., :vdim] = rnd(kv.shape[0], Hkv, vdim).to(BF16)
    q = (rnd(rows, H * dim) * 3.0).to(BF16)
    rel = 2 * rnd(reach, H)                                        # a row per distance
    table = hy.distance_table(rel, list(range(reach)), torch.zeros(H, device=DEV))
    cols = rnd(rows + 5, H * vdim).to(BF16)
    vp = hy.pad(vdim)
    rest = dict(G=G, softcap=softcap, chunk=chunk, weights=hy.KeyWeights(table, cols=cols, pitch=vdim).rows_from(5))
    c = hy.latent_gather(cache, bt, plan)
    outs = [hy.latent_prefill(q, c, c, plan, 0, scale, torch.zeros(rows, H * vp, dtype=BF16, device=DEV), H, dim, dvp, 0, 0, vdim, **rest)]
    if tc:
        k, vt = hy.gqa_gather(cache, bt, plan, Hkv, dim, dvp)
        outs.append(hy.latent_prefill_tc(q, k, vt, k, plan, 0, scale, torch.zeros_like(outs[0]), H, dim, dvp, 0, 0, vdim, **rest))
    row_seq = i32([i for i, (_, _, n) in enumerate(portions) for _ in range(n)])
    pos = i32([n0 + t for _, n0, n in portions for t in range(n)])
    seq_bt = bt[[s for s, _, _ in portions]].contiguous()
    dec = dict(softcap=softcap, weights=rest["weights"])
    for splits in (1, 4):
        outs.append(hy.gqa_decode(q, cache, seq_bt, row_seq, pos, i32([9] * 4), 0, chunk, scale, 1.0, torch.zeros_like(outs[0]), rows, H, Hkv, dim, vdim, dvp, splits, **dec))
    r0 = 0
    for s, n0, n in portions:
        p = torch.arange(n0 + n, device=DEV)
        flat = kv[(bt[s].long()[p // bs] * bs + p % bs)].double()
        K, V = flat[:, :Hkv * dim].view(-1, Hkv, dim), flat[:, Hkv * dim:].view(-1, Hkv, dvp)[..., :vdim]
        vis = p[None] <= p[n0:, None]
        vis &= p[None] // chunk == p[n0:, None] // chunk if chunk else True
        dist = (p[n0:, None] - p[None]).clamp(0, reach - 1)
        for h in range(H):
            sc = q[r0:r0 + n, h * dim:(h + 1) * dim].double() @ K[:, h // G].T * scale
            sc = softcap * torch.tanh(sc / softcap) if softcap else sc
            ref = (oracle.sigmoid(sc + rel.double()[dist, h]) * vis) @ V[:, h // G]
            ref = ref * oracle.sigmoid(cols[5 + r0:5 + r0 + n, h * vdim:(h + 1) * vdim].double())
            for o in outs:
                got = o[r0:r0 + n, h * vp:h * vp + vdim].double()
                assert ((got - ref).norm(dim=-1) / ref.norm(dim=-1)).max().item() < 2e-2
        r0 += n


@pytest.mark.parametrize("H,rank,rot", [(3, 48, 16), (20, 160, 32), (33, 512, 64)])
def test_sinks_in_latent_decoding(H, rank, rot):
    """Sinks from far below to far above the scores; the scalar form, the tile form, shared among splits."""
    from art_b200.ops import hybrid as hy

    rnd = rand(H)
    bs, n = 16, 300
    M, pitch = 6, 128
    for dt, tol in ((F32, 2e-5), (BF16, 2e-2)):
        cache = rnd(40, bs, rank + rot).to(dt)
        bt = torch.randperm(40, device=DEV)[:2 * 19].to(torch.int32).view(2, 19)
        ql, qr = rnd(H, pitch, rank).to(dt), rnd(H, pitch, rot).to(dt)
        row_seq, p = [0, 0, 1, 1, 0, 1], [0, 31, 32, 129, n - 1, 64]
        sink = torch.linspace(-30.0, 30.0, H, device=DEV)
        args = (ql, qr, cache, bt, i32(row_seq), i32(p), i32([n, n]), 0, 0.05)
        outs = [hy.latent_attend(*args, torch.zeros(H, pitch, rank, dtype=dt, device=DEV), M, sink=sink)]
        if dt == BF16:
            outs += [hy.latent_decode(*args, torch.zeros(H, pitch, rank, dtype=dt, device=DEV), M, s, sink=sink) for s in (1, 3, 7)]
        for m in range(M):
            t = torch.arange(p[m] + 1, device=DEV)
            c = cache.view(-1, rank + rot)[bt[row_seq[m]].long()[t // bs] * bs + t % bs].double()
            s = torch.cat([ql[:, m], qr[:, m]], -1).double() @ c.T * 0.05
            w = oracle.sink_softmax(s, sink.double()[:, None]) @ c[:, :rank]
            for o in outs:
                assert ((o[:, m].double() - w).norm(dim=-1) / w.norm(dim=-1).clamp(min=1e-3)).max().item() < tol


@pytest.mark.parametrize("H,dk,rot,dv,tiles", [(3, 48, 16, 40, False), (4, 64, 64, 56, True), (2, 128, 64, 128, True)])
def test_sinks_in_prompt_attention(H, dk, rot, dv, tiles):
    from art_b200.ops import hybrid as hy

    rnd = rand(dk)
    rank, n = 32, 290
    dvp = hy.prefill_tc_values(dk, rot, dv, 0.1) if tiles else hy.pad(dv, 16)
    plan = hy.plan_prefill([(0, 40, 250)], 0, DEV)
    nk = plan.n_keys
    q, k, v, c = rnd(250, H * (dk + rot)).to(BF16), rnd(nk, H * dk).to(BF16), rnd(nk, H * dvp).to(BF16), rnd(nk, rank + rot).to(BF16)
    sink = torch.linspace(-20.0, 25.0, H, device=DEV)
    vp = hy.pad(dv)
    kw = dict(weights=hy.KeyWeights(sink=sink))
    outs = [hy.latent_prefill(q, torch.cat([k, v], 1), c, plan, 0, 0.1, torch.zeros(250, H * vp, dtype=BF16, device=DEV), H, dk, dvp, rank, rot, dv, **kw)]
    if tiles:
        outs.append(hy.latent_prefill_tc(q, k, v.t().contiguous(), c, plan, 0, 0.1, torch.zeros_like(outs[0]), H, dk, dvp, rank, rot, dv, **kw))
    pos = torch.arange(n, device=DEV)
    for h in range(H):
        K = torch.cat([k[:n, h * dk:(h + 1) * dk], c[:n, rank:]], 1).double()
        s = (q[:, h * (dk + rot):(h + 1) * (dk + rot)].double() @ K.T * 0.1).masked_fill(pos[None] > pos[40:, None], -math.inf)
        ref = oracle.sink_softmax(s, sink.double()[h]) @ v[:n, h * dvp:h * dvp + dv].double()
        for o in outs:
            got = o[:, h * vp:h * vp + dv].double()
            assert ((got - ref).norm(dim=-1) / ref.norm(dim=-1).clamp(min=1e-6)).max().item() < 2e-2


@DTYPES
@pytest.mark.parametrize("H,Hkv,dim,vdim,rot", [(4, 2, 32, 24, 0), (4, 2, 32, 24, 16), (3, 3, 14, 22, 0), (2, 1, 6, 5, 2), (1, 1, 1, 1, 0), (24, 4, 128, 128, 0), (4, 0, 64, 64, 8),
                                                (100, 4, 256, 64, 0)])
def test_norms_of_each_head_and_column_gates_behind_the_projection(H, Hkv, dim, vdim, rot, dtype):
    from art_b200.ops import hybrid as hy

    rnd = rand(H)
    M, dk, dvp, nq, nk, nv = 7, hy.pad(dim, 16), hy.pad(vdim, 16), H * dim, Hkv * dim, Hkv * vdim
    pos, slot = [0, 1, 15, 16, 1000, 131071, 999999], [5, 40, -1, 0, 17, 63, 16]
    n = nq + nk + nv + H * vdim
    z = torch.zeros(M, hy.pad(n), device=DEV)
    z[:, :n] = 2 * rnd(M, n)
    wq, wk, temp = 1 + 0.3 * rnd(dim), 1 + 0.3 * rnd(dim), 0.5 + torch.rand(H, device=DEV)
    freq = torch.tensor([300.0 ** (-2 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64, device=DEV)
    for kind in (hy.KIND_F32 if dtype == F32 else hy.KIND_BF16, hy.KIND_TAKE):
        zz = z.to(BF16) if kind == hy.KIND_BF16 else z.clone()
        x = zz.double().cpu()
        cache = torch.full((4, 16, max(1, Hkv) * (dk + dvp)), 3.0, dtype=dtype, device=DEV)
        q = torch.full((M, H * dk), 9.0, dtype=dtype, device=DEV)
        vp = hy.pad(vdim)
        cols = torch.full((M, H * vp), 5.0, dtype=dtype, device=DEV) if kind == hy.KIND_TAKE else None
        hy.gqa_finish_norm(hy.Out(zz, kind), None, i32(slot), cache, q, H, Hkv, dim, vdim, dvp, wq, wk if Hkv else None, 1e-5,
                           hy.Rotation(rot, freq) if rot else None, i32(pos), None, True, temp, cols, vp if cols is not None else 0)

        def turned(y):
            src = y.clone()
            for i in range(rot // 2):
                ang = torch.tensor(pos, dtype=torch.float64) * float(freq[i])
                c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
                y[..., i], y[..., i + rot // 2] = src[..., i] * c - src[..., i + rot // 2] * s, src[..., i + rot // 2] * c + src[..., i] * s
            return y

        tol = 2e-5 if dtype == F32 else 2e-2
        want = turned(oracle.rms(x[:, :nq].view(M, H, dim), 1e-5) * wq.double().cpu() * temp.double().cpu()[:, None])
        got = q.view(M, H, dk).double().cpu()
        assert torch.allclose(got[..., :dim], want, atol=tol * 3, rtol=tol) and (dk == dim or float(got[..., dim:].abs().max()) == 0.0)
        rows = cache.view(64, -1).double().cpu()
        if Hkv:
            wk_ = turned(oracle.rms(x[:, nq:nq + nk].view(M, Hkv, dim), 1e-5) * wk.double().cpu())
            for m, sl in enumerate(slot):
                if sl >= 0:
                    assert torch.allclose(rows[sl, :Hkv * dk].view(Hkv, dk)[:, :dim], wk_[m], atol=tol * 3, rtol=tol)
                    assert torch.allclose(rows[sl, Hkv * dk:].view(Hkv, dvp)[:, :vdim], x[m, nq + nk:nq + nk + nv].view(Hkv, vdim), atol=tol, rtol=tol)
        assert float((rows[[i for i in range(64) if i not in slot or not Hkv]] - 3.0).abs().max()) == 0.0
        if cols is not None:
            assert torch.allclose(cols.view(M, H, vp)[..., :vdim].double().cpu(), x[:, nq + nk + nv:n].view(M, H, vdim), atol=tol, rtol=tol)
            assert float(zz[:, :n].abs().max()) == 0.0


@DTYPES
@pytest.mark.parametrize("H,dim,rot,rank", [(3, 20, 6, 36), (2, 16, 64, 48), (5, 8, 8, 24), (1, 2, 2, 1), (16, 128, 64, 512)])
def test_latent_finish_in_both_pairings(H, dim, rot, rank, dtype):
    from art_b200.ops import hybrid as hy

    rnd = rand(rot)
    M, n_abs = 6, 4
    pos, slot = [0, 3, 131071, 900000, 17, 999999], [5, -1, 0, 31, 8, 9]
    n = H * (dim + rot) + rank + rot
    dk, rot_p, rank_p = hy.pad(dim, 16), hy.pad(rot, 16), hy.pad(rank, 16)
    freq = torch.tensor([700.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=DEV)
    w = 1 + 0.2 * rnd(rank)
    for nxt in (False, True):
        for kind in (hy.KIND_F32 if dtype == F32 else hy.KIND_BF16, hy.KIND_TAKE):
            z = torch.zeros(M, hy.pad(n), device=DEV)
            z[:, :n] = rnd(M, n)
            zz = z.to(BF16) if kind == hy.KIND_BF16 else z.clone()
            x = zz.double().cpu()
            cache = torch.zeros(2, 16, rank_p + rot_p, dtype=dtype, device=DEV)
            qn, qr = (torch.zeros(H, 128, c, dtype=dtype, device=DEV) for c in (dk, rot_p))
            qe = torch.full((M - n_abs, H * (dk + rot_p)), 7.0, dtype=dtype, device=DEV)
            hy.latent_finish(hy.Out(zz, kind), w, hy.Rotation(rot, freq, 1.1, nxt), i32(pos), i32(slot), cache, n_abs, qn, qr, qe, H, dim, rank, 1e-5)

            def turned(y):
                out = y.clone()
                for i in range(rot // 2):
                    a, b = (2 * i, 2 * i + 1) if nxt else (i, i + rot // 2)
                    ang = torch.tensor(pos, dtype=torch.float64) * float(freq[i])
                    c, s = (1.1 * f(ang)[:, None] for f in (torch.cos, torch.sin))
                    out[..., a], out[..., b] = y[..., a] * c - y[..., b] * s, y[..., b] * c + y[..., a] * s
                return out

            tol = dict(atol=5e-6, rtol=2e-5) if dtype == F32 else dict(atol=2e-2, rtol=1e-2)
            q = x[:, :H * (dim + rot)].view(M, H, dim + rot)
            c = oracle.rms(x[:, H * (dim + rot):H * (dim + rot) + rank], 1e-5) * w.double().cpu()
            kr, tq = turned(x[:, None, H * (dim + rot) + rank:n])[:, 0], turned(q[..., dim:])
            for m in range(M):
                if slot[m] >= 0:
                    row = cache.view(32, -1)[slot[m]].double().cpu()
                    assert torch.allclose(row[:rank], c[m], **tol) and torch.allclose(row[rank_p:rank_p + rot], kr[m], **tol)
                if m < n_abs:
                    a, b = qn[:, m].double().cpu(), qr[:, m].double().cpu()
                else:
                    e = qe[m - n_abs].view(H, dk + rot_p).double().cpu()
                    a, b = e[:, :dk], e[:, dk:]
                assert torch.allclose(a[:, :dim], q[m, :, :dim], **tol) and torch.allclose(b[:, :rot], tq[m], **tol)
                assert float(a[:, dim:].abs().sum() + b[:, rot:].abs().sum()) == 0.0
            assert kind != hy.KIND_TAKE or float(zz[:, :n].abs().max()) == 0.0


def test_router_chooses_among_the_best_groups():
    from art_b200.ops import moe as ops

    for E, groups, keep, k, scale in ((8, 4, 3, 4, 2.0), (12, 3, 1, 4, 0.5), (66, 11, 2, 7, 1.0), (256, 8, 4, 16, 2.5), (10, 1, 1, 3, 1.5), (6, 6, 2, 2, 1.0), (9, 3, 3, 2, 1.0)):
        z = rand(E)(41, E)
        z[3] = z[3, 0]                                            # all alike: the first ones
        z[4, E - 1] = 40.0                                        # a group for the sake of its largest one, whose neighbours are small
        z[4, E - E // groups:E - 1] -= 5.0
        ws = torch.cat([z, torch.full((41, 5), 3.0, device=DEV)], 1)
        plan = ops.route(ws[:, :E], k, False, take=True, groups=groups, keep=keep, scale=scale)
        best, a = oracle.route(torch.eye(41, dtype=torch.float64), {"router": z.double().cpu().T}, {"groups": {"count": groups, "keep": keep}, "top": k, "scale": scale})
        assert torch.equal(plan.topi.cpu().long(), best) and torch.allclose(plan.topw.cpu().double(), a, atol=1e-6)
        assert float(ws[:, :E].abs().max()) == 0.0 and float((ws[:, E:] - 3.0).abs().max()) == 0.0
        assert int(plan.counts.sum()) == 41 * k


@DTYPES
@pytest.mark.parametrize("experts,groups,keep,top,ff", [(8, 4, 2, 3, 16), (1, 1, 1, 1, 20), (40, 8, 3, 6, 33), (256, 16, 4, 16, 16), (6, 2, 1, 3, 7)])
def test_mixture_of_experts_alone(experts, groups, keep, top, ff, dtype):
    """The gated feed-forward of a layer against the equations; bf16 rows are compared where the choice is no close call."""
    from art_b200.engine.runner import SeqView
    from art_b200.ops import hybrid as hy

    p = group_moe(experts, groups, keep, top, ff, 1.3)
    d = one(sigmoid_heads(mlp=p))
    run = session(d, dtype).runner
    W = {k[len("l0."):]: t.double() for k, t in model(d)[1].items() if k.startswith("l0.")}
    x = torch.zeros(75, run.dp, device=DEV)
    x[:, :68] = rand(2)(75, 68).to(dtype).float()
    h = x.to(dtype)
    b = run._pack([SeqView(tokens(75, 97), 0, [0, 1, 2, 3, 4], -1, 0.0, 0, 0)])[0]
    out = torch.zeros_like(x)
    hy.residual_step(out, None, 68, 1e-5, sub=run._mlp_moe(run.cfg.layers[0], run.layers[0], x, h, b), x_in=torch.zeros_like(x))
    hh = h[:, :68].double().cpu()
    ref = oracle.moe(hh, oracle.part(W, "mlp"), p) * oracle.sigmoid(hh @ W["rg2"].T + W["rg2.b"])
    s = torch.softmax(hh @ W["mlp.router"].T, -1).view(75, groups, -1)
    g = s.amax(-1).sort(-1, descending=True).values
    best = s.amax(-1) >= g[:, keep - 1:keep]
    e = s.masked_fill(~best[..., None], -1.0).flatten(1).sort(-1, descending=True).values
    clear = torch.ones(75, dtype=torch.bool)
    if keep < groups:
        clear &= g[:, keep - 1] - g[:, keep] > 1e-3 * g[:, keep - 1]
    if top < experts:
        clear &= e[:, top - 1] - e[:, top] > 1e-3 * e[:, top - 1]
    err = ((out[:, :68].cpu().double() - ref).norm(dim=-1) / ref.norm(dim=-1))[clear]
    assert int(clear.sum()) > 40 and float(err.max()) < (1e-5 if dtype == F32 else 2e-2)


@DTYPES
@pytest.mark.parametrize("d,n_in,n_out", [(101, 1, 2), (64, 2, 2), (1030, 2, 1), (2500, 3, 3), (516, 4, 4), (4096, 2, 2), (96, 1, 1), (5000, 8, 8), (40, 7, 1), (9000, 3, 3)])
def test_stream_step_mixes_all_copies_at_once(d, n_in, n_out, dtype):
    """Results as products, expert rows or both, every kind of gate; in place where the number of copies stays."""
    from art_b200.ops import hybrid as hy

    rnd = rand(d)
    dp, M, r = hy.pad(d), 5, slice(0, d)

    def padded(*shape):
        t = torch.zeros(*shape[:-1], dp, device=DEV)
        t[..., r] = rnd(*shape[:-1], d)
        return t

    for kind in (hy.KIND_F32, hy.KIND_TAKE) + ((hy.KIND_BF16,) if dtype == BF16 else ()):
        xs, y, gate, rows = padded(M, n_in, d), padded(M, d), padded(M, d), padded(20, d).to(dtype)
        bias, w, coef = padded(d), padded(d), rnd((n_in + 2) * n_out)
        pos, wt = torch.randint(0, 20, (M, 3), device=DEV).int(), rnd(M, 3)
        mix, o, nxt = coef[:n_in * n_out].view(n_in, n_out).double(), coef[-2 * n_out:-n_out].double(), coef[-n_out:].double()
        for form in ("y", "rows", "both"):
            yy, gg = (t.to(BF16) if kind == hy.KIND_BF16 else t.clone() for t in (y, gate))
            ref = yy.double() if form != "rows" else torch.zeros_like(y).double()
            if form != "y":
                ref = ref + (wt.double()[..., None] * rows.double()[pos.long()]).sum(1)
            ref = ref * oracle.sigmoid(gg.double() + bias.double())
            x_in = xs.reshape(M, n_in * dp).clone()
            x_out = x_in if n_in == n_out else torch.full((M, n_out * dp), 9.0, device=DEV)
            h = torch.empty(M, dp, dtype=dtype, device=DEV)
            sub = hy.Sublayer(hy.Out(yy, kind) if form != "rows" else None, col_gate=hy.Out(gg, kind), col_bias=bias)
            if form != "y":
                sub.rows, sub.pos, sub.weight = rows, pos, wt
            hy.residual_step(x_out, None, d, 1e-5, sub=sub, x_in=x_in, w_next=w, h=h, streams=hy.Streams(n_in, n_out, coef))
            want = torch.einsum("mid,io->mod", xs.double(), mix) + o[None, :, None] * ref[:, None]
            assert torch.allclose(x_out.view(M, n_out, dp).double(), want, atol=1e-4, rtol=1e-4)
            u = torch.einsum("mod,o->md", want, nxt)
            hw = torch.zeros(M, dp, dtype=torch.float64, device=DEV)
            hw[:, r] = oracle.rms(u[:, r], 1e-5) * w[r].double()
            assert torch.allclose(h.double(), hw, atol=1e-4 if dtype == F32 else 3e-2, rtol=1e-4 if dtype == F32 else 1e-2)
            if kind == hy.KIND_TAKE:
                assert float(gg.abs().max()) == 0.0 and (form == "rows" or float(yy.abs().max()) == 0.0)


@DTYPES
def test_embedding_of_streams_and_gates_of_a_single_stream(dtype):
    from art_b200.ops import hybrid as hy

    rnd = rand(0)
    d, dp = 70, 72
    table, w = torch.zeros(11, dp, device=DEV), torch.zeros(dp, device=DEV)
    table[:, :d], w[:d] = rnd(11, d), rnd(d)
    table = table.to(dtype)
    toks = torch.tensor([3, 0, 10], device=DEV)
    x, h = torch.zeros(3, dp, device=DEV), torch.empty(3, dp, dtype=dtype, device=DEV)
    hy.residual_step(x, None, d, 1e-5, tokens=toks, table=table, w_next=w, h=h, streams=hy.Streams(0, 1, torch.tensor([1.0, -0.7], device=DEV)))
    e = table.double()[toks]
    assert torch.equal(x, table.float()[toks])
    assert torch.allclose(h[:, :d].double(), oracle.rms(-0.7 * e[:, :d], 1e-5) * w[:d].double(), atol=1e-5 if dtype == F32 else 2e-2, rtol=1e-2)
    y, g, b = torch.zeros(3, dp, device=DEV), torch.zeros(3, dp, device=DEV), torch.zeros(dp, device=DEV)
    y[:, :d], g[:, :d], b[:d] = rnd(3, d), rnd(3, d), rnd(d)
    x2 = x.clone()
    hy.residual_step(x2, None, d, 1e-5, sub=hy.Sublayer(hy.as_out(y), col_gate=hy.as_out(g), col_bias=b), x_in=x, mult=0.5)
    assert torch.allclose(x2.double(), e + 0.5 * y.double() * oracle.sigmoid(g.double() + b.double()), atol=1e-5)
    with pytest.raises(ValueError):
        hy.residual_step(x2, None, d, 1e-5, y=hy.as_out(y), x_in=x, streams=hy.Streams(2, 1, torch.zeros(4, device=DEV)))
    with pytest.raises(ValueError):
        hy.residual_step(x2, w, d, 1e-5, sub=hy.Sublayer(hy.as_out(y), col_gate=hy.as_out(g), col_bias=b), x_in=x)


@pytest.mark.parametrize("M,N,first,pairs", [(40, 136, 72, False), (300, 264, 8, False), (300, 512, 512, False), (1030, 520, 200, True)])
def test_squared_relu_of_the_first_columns(M, N, first, pairs):
    from art_b200.ops.gemm import gemm_tn

    rnd = rand(N)
    a, W = rnd(M, 128).to(BF16), rnd(N, 128).mul(0.2).to(BF16)
    ref = a.double() @ W.double().T
    ref[:, :first] = oracle.relu2(ref[:, :first])
    assert torch.allclose(gemm_tn(a, W, relu2=True, relu2_cols=first, two_cta=pairs).double(), ref, atol=1e-2, rtol=1e-2)


@DTYPES
def test_greedy_generation_through_the_engine(dtype):
    """More requests than the batch holds, prompts in portions beside decoding, shared prefixes from the block cache,
    multi-step decoding with captured graphs; fp32 must reproduce the oracle's greedy tokens, bf16 (dense feed-forwards: no
    close calls of a router) its log-probabilities."""
    from art_b200.engine.engine import SamplingParams
    from art_b200.engine.factory import build_engine
    from art_b200.models.config import config_from_dict

    d = small_gaparax()
    if dtype == BF16:
        for e in d["layers"]:
            e["mlp"] = relu2_dense(40) if e["mlp"] else None
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
def test_long_decoding_passes_over_pages_and_chunks(dtype):
    d = gaparax([sigmoid_heads(heads=2, kv_heads=1, chunk=50, bias_max=30), sink_latent(mlp=relu2_dense()), sigmoid_heads(heads=2, chunk=128, bias_max=100)], vocab=61, width=64)
    toks = tokens(270, 61, 8)
    check(feed(session(d, dtype), toks, [9, 1]), want_logits(d, toks), dtype, 1.5)


@DTYPES
def test_batched_decoding_with_split_products_and_workspaces(dtype):
    """Wide enough that decode products are split and taken by the kernels behind them; several sequences, every step a
    single token each, against each prompt alone."""
    d = gaparax([sigmoid_heads(heads=4, kv_heads=2, dim=64, vdim=72, chunk=24, scale=0.125, mlp=relu2_dense(640)), sink_latent(heads=4, dim=64, rot=64, rank=128, vdim=64, scale=0.1,
                 mlp=group_moe(6, 2, 2, 6, 64)), sigmoid_heads(heads=8, kv_heads=1, dim=32, vdim=20, chunk=33)], vocab=304, width=512, streams=2)
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


@DTYPES
@pytest.mark.parametrize("rows,reach", [(2, 2), (6, 300), (64, 40)])
def test_distance_tables_of_other_sizes(rows, reach, dtype):
    """The rows of a table are its tensor's: few and many, buckets that end before and behind the chunk."""
    d = one(sigmoid_heads(chunk=90, bias_max=reach), sigmoid_heads(heads=2, dim=64, vdim=64, chunk=200, bias_max=reach))
    w = dict(model(d)[1])
    for i, h in ((0, 4), (1, 2)):
        w[f"l{i}.mix.rel"] = torch.randn(rows, h, generator=torch.Generator().manual_seed(rows)).mul(2).to(BF16)
    toks = tokens(230, 97, 6)
    if reach <= rows // 2:
        w["l0.mix.rel"], w["l1.mix.rel"] = w["l0.mix.rel"][:20], w["l1.mix.rel"][:30]
    want = oracle.forward(d, w, toks, torch.float64).float()
    rep = session(d, dtype, weights=w)
    for cuts in ([230], [100, 1], [37]):
        check(feed(rep, toks, cuts), want, dtype)


def test_trace_command_line(tmp_path):
    import numpy as np
    from safetensors.torch import save_file

    d = small_gaparax()
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

    cfg = resolve_config("gaparax-tiny")
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
