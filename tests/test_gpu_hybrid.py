"""Hybrid decoders on the GPU against the plain oracle: each mixer alone and whole models, in fp32 and bf16, as whole prompts,
token by token, in portions, in mixed batches and through the engine's own generation."""
import json
import os
import subprocess
import sys

import pytest
import torch

from . import nikelix_oracle as oracle
from .hybrid_models import aligned_design, design, hgrn2, latent, single_layer, small_design, wkv
from .hybrid_session import BF16, DEV, F32, check, feed, mixed_session, model, session, tokens, want_logits

pytestmark = pytest.mark.gpu


@pytest.fixture(autouse=True)
def _status_clean():
    yield
    from art_b200.ops import _lib

    torch.cuda.synchronize()
    _lib.check_status()


LAYERS = {"latent": latent(), "latent-one": latent(heads=1, dim=8, rot=2, rank=8, vdim=8, window=1), "latent-wide": latent(heads=17, dim=40, rot=16, rank=144, vdim=136),
          "latent-blocks": latent(heads=2, dim=64, rot=64, rank=80, vdim=72, window=33), "latent-full": latent(heads=2, window=0), "hgrn2": hgrn2(), "hgrn2-one": hgrn2(heads=1, dim=1, vdim=5), "hgrn2-wide": hgrn2(heads=2, dim=130, vdim=100),
          "wkv": wkv(), "wkv-one": wkv(heads=1, dim=4), "wkv-wide": wkv(heads=2, dim=200), "no-mlp": wkv(ff=0)}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(LAYERS))
def test_one_layer_prompts_portions_and_decoding(name, dtype):
    d = single_layer(LAYERS[name])
    toks = tokens(75 if name != "latent-blocks" else 290, 97, 1)
    if name == "latent-full":      # the oracle reads the same dictionary: a window longer than the sequence stands for none
        want = oracle.forward(single_layer(latent(heads=2, window=10 ** 6)), model(d)[1], toks, torch.float64).float()
    else:
        want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([300], [1], [40, 1], [2], [17, 2, 33, 3]):
        check(feed(rep, toks, cuts), want, dtype)
    assert rep.bm.num_free == 64


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("which", ["small", "aligned"])
def test_whole_model_every_cut(which, dtype):
    d = small_design() if which == "small" else aligned_design()
    toks = tokens(330 if which == "aligned" else 140, d["vocab"], 2)
    want = want_logits(d, toks)
    rep = session(d, dtype)
    for cuts in ([len(toks)], [len(toks) - 40, 1], [2, 64, 3, 16, 5, 31], [128, 17]):
        check(feed(rep, toks, cuts), want, dtype, 1.5)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_residual_stream_after_every_layer(dtype):
    from art_b200.engine.runner import SeqView

    d = small_design()
    toks = tokens(33, d["vocab"], 3)
    ref = []
    oracle.forward(d, model(d)[1], toks, torch.float64, ref)
    run = session(d, dtype).runner
    got = run.layer_outputs([SeqView(toks, 0, [5, 2, 9], -1, 0.0, 0, 0, state_slot=3)])
    assert len(got) == len(ref) == len(d["layers"])
    for a, b in zip(got, ref):
        assert ((a.cpu() - b).norm() / b.norm()).item() < (1e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_requests_in_mixed_batches_reuse_pages_and_slots(dtype):
    mixed_session(aligned_design(), dtype, [180, 1, 37, 250, 90, 64, 33, 2], check)


def test_far_past_is_kept_by_the_states_and_cut_by_the_window():
    """One changed token shows exactly as far as it must: through the recurrent layers at any distance, through a window of
    w keys only up to w - 1 positions later (one layer), in prompts and in decoding."""
    toks = tokens(90, 97, 6)
    other = list(toks)
    other[20] = (toks[20] + 31) % 97
    for layer, reach in ((latent(window=24), 23), (latent(window=17, heads=1), 16), (hgrn2(), 69), (wkv(), 69)):
        d = single_layer(layer)
        for cuts in ([90], [50, 1], [30, 7]):
            rep = session(d, F32)
            diff = (feed(rep, toks, cuts) - feed(rep, other, cuts)).abs().amax(-1)
            seen = (diff > 0).nonzero().flatten().tolist()
            assert seen[0] == 20 and (seen[-1] == 20 + reach if layer["type"] == "latent_attention" else seen[-1] > 60), (layer["type"], seen[-1])


@pytest.mark.parametrize("form", ["scalar32", "scalar16", "decode", "decode-split", "prefill"])
@pytest.mark.parametrize("window", [1, 16, 50, 64, 129])
def test_window_edges_and_page_borders_of_every_attention_form(form, window):
    """A key whose score towers above all others sits just inside, then just outside the window of one query; the query's
    output must be that key's latent, then must not contain it.  Pages are shuffled, positions lie around page borders."""
    from art_b200.ops import hybrid as hy

    H, rank, rot, bs, n = 3, 32, 16, 16, 200
    dt = F32 if form == "scalar32" else BF16
    g = torch.Generator(device=DEV).manual_seed(window)
    rnd = lambda *s: torch.randn(*s, device=DEV, generator=g)      # noqa: E731
    pages = torch.randperm(20, device=DEV, generator=g)[:13].to(torch.int32)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)      # noqa: E731
    for p in (0, 15, 16, 17, 63, 64, 127, 128, 150, 199):
        for inside in (True, False):
            j = p - window + 1 if inside else p - window
            if j < 0:
                continue
            cache = torch.zeros(20, bs, rank + rot, device=DEV)
            flat = 0.1 * rnd(n, rank + rot)
            q = rnd(H, rank + rot)
            q = q / q.norm(dim=-1, keepdim=True)
            flat[j] += 40.0 * q.sum(0)
            for t in range(n):
                cache[pages[t // bs], t % bs] = flat[t]
            cache = cache.to(dt)
            lo = max(0, p - window + 1)
            K = flat[lo:p + 1].to(dt).double()
            a = torch.softmax(q.to(dt).double() @ K.T, -1)
            want = (a @ K[:, :rank]).float()
            bt = pages.view(1, -1).contiguous()
            if form == "prefill":
                # identity expansion: keys are the latents, values their first `rank` columns
                plan = hy.plan_prefill([(0, p, 1)] if window > 1 else [(0, p, 1)], window, DEV)
                c = hy.latent_gather(cache, bt, plan)
                kv = torch.cat([c[:, :rank]] * H + [c[:, :rank]] * H, 1).contiguous()
                o = torch.zeros(1, H * rank, dtype=dt, device=DEV)
                hy.latent_prefill(q.to(dt).reshape(1, -1), kv, c, plan, window, 1.0, o, H, rank, rank, rank, rot, rank)
                got = o.view(H, rank)
            else:
                ql, qr = torch.zeros(H, 128, rank, dtype=dt, device=DEV), torch.zeros(H, 128, rot, dtype=dt, device=DEV)
                ql[:, 0], qr[:, 0] = q[:, :rank].to(dt), q[:, rank:].to(dt)
                o = torch.zeros_like(ql)
                args = (ql, qr, cache, bt, i32([0]), i32([p]), i32([p + 1]), window, 1.0, o, 1)
                if form.startswith("scalar"):
                    hy.latent_attend(*args)
                else:
                    hy.latent_decode(*args, splits=3 if form == "decode-split" else 1)
                got = o[:, 0]
            err = (got.float() - want).norm() / want.norm()
            assert float(err) < (1e-5 if dt == F32 else 2e-2), (p, inside, float(err))


@pytest.mark.parametrize("H,dk,rot,rank,vdim,window", [(2, 48, 16, 32, 40, 100), (1, 128, 64, 64, 128, 300), (3, 16, 16, 16, 8, 1), (2, 64, 32, 48, 96, 0),
                                                       (2, 128, 64, 96, 128, 129), (3, 64, 64, 32, 56, 1), (2, 64, 0, 32, 128, 0), (1, 128, 0, 16, 72, 500),
                                                       (2, 128, 64, 64, 64, 250)])
def test_prefill_attention_tiles_against_plain_softmax(H, dk, rot, rank, vdim, window):
    """Several query tiles, sequences that continue a cached prefix, ragged ends, values narrower than the tile; both forms
    of the kernel where the sizes suit both."""
    from art_b200.ops import hybrid as hy

    g = torch.Generator(device=DEV).manual_seed(0)
    dv = hy.pad(vdim, 16)
    portions = [(1, 0, 130), (0, 77, 257), (2, 300, 20), (3, 1, 17)]
    plan = hy.plan_prefill(portions, window, DEV)
    rows = sum(n for _, _, n in portions)
    rnd = lambda *s: torch.randn(*s, device=DEV, generator=g).to(BF16)      # noqa: E731
    q, kv, c = 1.5 * rnd(rows, H * (dk + rot)), rnd(plan.n_keys, H * (dk + dv)), rnd(plan.n_keys, rank + rot)
    outs = []
    if rot:
        o = torch.zeros(rows, H * hy.pad(vdim), dtype=BF16, device=DEV)
        outs.append(hy.latent_prefill(q, kv, c, plan, window, 0.11, o, H, dk, dv, rank, rot, vdim))
    tdv = hy.prefill_tc_values(dk, rot, vdim, 0.11)
    assert bool(tdv) == (dk % 64 == 0 and rot % 64 == 0)
    if tdv:
        v = torch.zeros(H, tdv, plan.n_keys, dtype=BF16, device=DEV)
        v[:, :dv] = kv[:, H * dk:].reshape(-1, H, dv).permute(1, 2, 0)
        o = torch.zeros(rows, H * hy.pad(vdim), dtype=BF16, device=DEV)
        outs.append(hy.latent_prefill_tc(q, kv[:, :H * dk].contiguous(), v.view(H * tdv, -1), c, plan, window, 0.11, o, H, dk, tdv, rank, rot, vdim))
    r0 = 0
    for i, (_, n0, n) in enumerate(portions):
        k0, kp = int(plan.key_off[i]), int(plan.key_pos0[i])
        nk = n0 + n - kp
        pos, kpos = torch.arange(n0, n0 + n, device=DEV), torch.arange(kp, kp + nk, device=DEV)
        vis = kpos[None] <= pos[:, None]
        if window:
            vis &= kpos[None] > pos[:, None] - window
        for h in range(H):
            Q = q[r0:r0 + n, h * (dk + rot):(h + 1) * (dk + rot)].float()
            K = torch.cat([kv[k0:k0 + nk, h * dk:(h + 1) * dk], c[k0:k0 + nk, rank:]], 1).float()
            V = kv[k0:k0 + nk, H * dk + h * dv:H * dk + h * dv + vdim].float()
            ref = torch.softmax((Q @ K.T * 0.11).masked_fill(~vis, float("-inf")), -1) @ V
            for o in outs:
                got = o[r0:r0 + n, h * hy.pad(vdim):h * hy.pad(vdim) + vdim].float()
                assert ((got - ref).norm(dim=-1) / ref.norm(dim=-1)).max().item() < 2e-2
        r0 += n


@pytest.mark.parametrize("mode", ["hgrn2", "wkv"])
@pytest.mark.parametrize("n_seqs,H,dim,vdim", [(1, 1, 4, 4), (1, 2, 33, 20), (40, 4, 128, 128), (90, 2, 64, 64), (3, 2, 256, 96), (160, 1, 96, 40)])
def test_linear_scan_and_decode_kernels_against_the_recurrence(mode, n_seqs, H, dim, vdim):
    """Every slice width of the scan kernel; strong and weak decays; portions of several lengths from given states, then one
    decoded token per sequence."""
    from art_b200.ops import hybrid as hy

    wkv_mode = mode == "wkv"
    vdim = dim if wkv_mode else vdim
    g = torch.Generator(device=DEV).manual_seed(dim)
    rnd = lambda *s: torch.randn(*s, device=DEV, generator=g)      # noqa: E731
    lens = [(i * 7) % 37 + 1 for i in range(n_seqs)]
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    M, n = cu[-1], H * dim
    q, k, v = rnd(M, n).to(BF16), rnd(M, n).to(BF16), rnd(M, H * vdim).to(BF16)
    gr, bias, aux = 3 * rnd(M, n), rnd(n), torch.rand(n, device=DEV, generator=g)
    ld = hy.pad(dim, 4)
    state = torch.zeros(n_seqs + 1, H, vdim, ld, device=DEV)
    state[..., :dim] = rnd(n_seqs + 1, H, vdim, dim)
    s0 = state.clone()
    fresh = [i % 3 == 0 for i in range(n_seqs)]
    slots = list(range(n_seqs, 0, -1))
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)      # noqa: E731
    ctx = [n_ if f else n_ + 5 for n_, f in zip(lens, fresh)]
    o = torch.zeros(M, H * vdim, device=DEV)
    m = hy.SCAN_WKV if wkv_mode else hy.SCAN_HGRN2
    as_ = hy.as_out
    hy.linear_scan(m, as_(q), as_(k) if wkv_mode else None, as_(v), as_(gr), bias, aux, state, i32(cu), i32(ctx), i32(slots), n_seqs, H, dim, vdim, o)

    def gates(rows):
        qq, kk, vv = (t[rows].double().view(-1, H, w) for t, w in ((q, dim), (k, dim), (v, vdim)))
        z = (gr[rows] + bias).double().view(-1, H, dim)
        a = aux.double().view(H, dim)
        if wkv_mode:
            return qq, kk, vv, torch.exp(-torch.exp(z)), a
        f = a + (1 - a) * torch.sigmoid(z)
        return oracle.silu(qq), 1 - f, vv, f, a

    def step(S, qt, kt, vt, ft, a):
        kv = kt.unsqueeze(-1) * vt.unsqueeze(-2)
        new = ft.unsqueeze(-1) * S + kv
        read = S + a.unsqueeze(-1) * kv if wkv_mode else new
        return new, torch.einsum("...kv,...k->...v", read, qt)

    def close(a, b):
        assert ((a.double() - b).norm() / (b.norm() + 1e-9)).item() < 2e-6

    for i in list(range(min(n_seqs, 6))) + [n_seqs - 1]:
        qq, kk, vv, f, a = gates(slice(cu[i], cu[i + 1]))
        S = torch.zeros(H, dim, vdim, dtype=torch.float64, device=DEV) if fresh[i] else s0[slots[i], ..., :dim].double().transpose(1, 2)
        for t in range(lens[i]):
            S, ot = step(S, qq[t], kk[t], vv[t], f[t], a)
            close(o[cu[i] + t].view(H, vdim), ot)
        close(state[slots[i], ..., :dim].transpose(1, 2), S)
    assert torch.equal(state[0], s0[0])                      # a slot nobody holds stays as it is
    # one token each, the last sequence being a padding row
    d = n_seqs
    before = state.clone()
    sl = slots[:-1] + [-1] if n_seqs > 1 else slots
    w, vp = rnd(H * vdim), hy.pad(vdim)
    gate = rnd(d, H * vdim).to(BF16)
    out = torch.zeros(d, H * vp, device=DEV)
    f32 = lambda t: as_(t[:d].float().contiguous())      # noqa: E731
    hy.linear_decode(m, f32(q), f32(k) if wkv_mode else None, f32(v), as_(gr[:d].contiguous()), bias, aux, state, i32(list(range(d + 1))), i32([9] * d),
                     i32(sl), H, dim, vdim, w, True, as_(gate), out, vp, 1e-5)
    qq, kk, vv, f, a = gates(slice(0, d))
    for i in range(min(d, 5)):
        if sl[i] < 0:
            continue
        S, ot = step(before[sl[i], ..., :dim].double().transpose(1, 2), qq[i], kk[i], vv[i], f[i], a)
        y = oracle.rms(ot, 1e-5).reshape(-1) * w.double() * oracle.silu(gate[i].double())
        close(out[i].view(H, vp)[:, :vdim].reshape(-1), y)
        close(state[sl[i], ..., :dim].transpose(1, 2), S)


def test_poly_norm_token_shift_and_depth_average_rows():
    from art_b200.ops import hybrid as hy

    g = torch.Generator(device=DEV).manual_seed(1)
    rnd = lambda *s: torch.randn(*s, device=DEV, generator=g)      # noqa: E731
    for n in (1, 75, 384, 2500, 9000):
        z = torch.zeros(7, hy.pad(n), device=DEV)
        z[:, :n] = 2 * rnd(7, n)
        act = torch.tensor([0.7, -0.4, 0.3, 0.11], device=DEV)
        ws = z.clone()
        out = torch.full_like(z, 9.0)
        hy.poly_norm(hy.Out(ws, hy.KIND_TAKE), act, out, n, 1e-4)
        ref = oracle.poly_norm(z[:, :n].double(), act.double(), 1e-4)
        assert ((out[:, :n].double() - ref).norm() / ref.norm()).item() < 1e-5
        assert float(out[:, n:].abs().sum()) == 0.0 and float(ws.abs().max()) == 0.0      # padding zero, workspace handed back zero
    d, dp, M, L = 100, 104, 5, 4
    hist = torch.zeros(L + 2, M, dp, device=DEV)
    hist[:L, :, :d] = rnd(L, M, d)
    x0, y, w, w2 = (torch.zeros(*s, device=DEV) for s in ((M, dp), (M, dp), (dp,), (dp,)))
    x0[:, :d], y[:, :d], w[:d], w2[:d] = rnd(M, d), rnd(M, d), rnd(d), rnd(d)
    avg = rnd(L + 1)
    x, h = torch.empty(M, dp, device=DEV), torch.empty(M, dp, device=DEV)
    hy.residual_step(x, w, d, 1e-5, y=hy.as_out(y), x_in=x0, mult=0.3, hist=hist, hist_n=L, avg=avg, w_next=w2, h=h)
    new = x0[:, :d].double() + 0.3 * oracle.rms(y[:, :d].double(), 1e-5) * w[:d].double()
    ref = sum(avg[j].double() * (hist[j, :, :d].double() if j < L else new) for j in range(L + 1))
    assert torch.allclose(hist[L, :, :d].double(), new, atol=1e-5) and torch.allclose(x[:, :d].double(), ref, atol=1e-5)
    assert torch.allclose(h[:, :d].double(), oracle.rms(ref, 1e-5) * w2[:d].double(), atol=1e-5) and float(h[:, d:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_greedy_generation_through_the_engine(dtype):
    """More requests than state slots, prompts in portions beside decoding, multi-step decoding with captured graphs; fp32
    must reproduce the oracle's greedy tokens, bf16 its log-probabilities up to near-ties."""
    from art_b200.engine.engine import SamplingParams
    from art_b200.engine.factory import build_engine
    from art_b200.models.config import config_from_dict

    d = small_design()
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
    import asyncio

    got = asyncio.run(eng.score(prompts[1], seqs[1].output_ids[:6]))
    assert all(abs(a - b) < (1e-3 if dtype == F32 else 0.1) for a, b in zip(got, seqs[1].logprobs[:6]))
    sampled = eng.generate_sync(prompts[0], SamplingParams(max_tokens=8, temperature=0.9, top_k=5, top_logprobs=3, seed=1))
    assert len(sampled.output_ids) == 8 and all(len(t) == 3 for t in sampled.top_logprobs)
    eng.runner.close()


def test_long_decoding_passes_over_windows_and_pages():
    """A few hundred decoded tokens: every page border and window edge is crossed while decoding."""
    d = design([latent(window=40), hgrn2(), wkv()], vocab=61, width=64)
    toks = tokens(260, 61, 8)
    want = want_logits(d, toks)
    for dtype in (F32, BF16):
        check(feed(session(d, dtype), toks, [9, 1]), want, dtype, 1.5)


def test_trace_command_line(tmp_path):
    from safetensors.torch import save_file

    d = small_design()
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
    for dtype in ("float32", "bfloat16"):
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                           input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=180)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
        for step, rows in ((0, [0, 29]), (2, [39, 2])):
            import numpy as np

            got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").copy()).view(len(rows), d["vocab"])
            check(got, ref[rows], F32 if dtype == "float32" else BF16)
            (tmp_path / f"{step}.f32").unlink()
    assert sys.executable


def test_completion_server_over_a_hybrid_model():
    """The OpenAI server on the preset engine: chat, logit processing, structured output; adapters are refused."""
    import asyncio

    import httpx

    from art_b200.engine.factory import build_engine
    from art_b200.engine.server import OpenAIServer
    from art_b200.local.tokenizer import ByteChatTokenizer
    from art_b200.models.config import resolve_config
    from art_b200.models.weights import init_base_weights

    cfg = resolve_config("nikelix-tiny")
    tok = ByteChatTokenizer(cfg.vocab_size)
    eng = build_engine(cfg, init_base_weights(cfg, dtype=BF16, device=DEV), num_blocks=64, max_num_seqs=4, eos_token_id=tok.eos_token_id)
    eng.start()
    srv = OpenAIServer(eng, tok, "nikelix-tiny")

    async def main():
        async with httpx.AsyncClient(transport=httpx.ASGITransport(app=srv.app), base_url="http://t", headers={"Authorization": "Bearer default"}) as c:
            body = {"model": "nikelix-tiny", "messages": [{"role": "user", "content": "hi"}], "max_tokens": 6, "n": 3, "seed": 1}
            r = await c.post("/v1/chat/completions", json=body)
            assert r.status_code == 200 and len(r.json()["choices"]) == 3
            r = await c.post("/v1/chat/completions", json={**body, "n": 1, "frequency_penalty": 0.5, "top_p": 0.8})
            assert r.status_code == 200
            r = await c.post("/v1/chat/completions", json={**body, "n": 1, "guided_choice": ["yes", "no"]})
            assert r.json()["choices"][0]["message"]["content"] in ("yes", "no")

    try:
        asyncio.run(asyncio.wait_for(main(), 30))
        assert eng.error is None
        with pytest.raises(ValueError, match="adapters"):
            eng.runner.set_adapter(0, {})
        assert eng.state_slots.num_free + len(eng.running) == 4
    finally:
        eng.shutdown()
        eng.runner.close()
