"""What the GPU tests of the hybrid designs share: random models, the oracle's logits, a replay session, comparisons."""
import functools
import json

import torch

from . import gaborax_oracle, gaparax_oracle, naselorn_oracle, nikelix_oracle

DEV = "cuda"
F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 2e-5, BF16: 4e-2}          # root mean square over the vocabulary, relative to that of the oracle's logits
ORACLES = {"Nikelix": nikelix_oracle, "Naselorn": naselorn_oracle, "Gaborax": gaborax_oracle, "Gaparax": gaparax_oracle}


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@functools.lru_cache(maxsize=None)
def _model(key, seed):
    from art_b200.models.config import config_from_dict
    from art_b200.models.hybrid import init_hybrid_weights

    d = json.loads(key)
    return d, init_hybrid_weights(config_from_dict(d), seed=seed, dtype=BF16)


def model(d, seed=0):
    return _model(json.dumps(d), seed)


@functools.lru_cache(maxsize=None)
def _oracle(key, seed, toks):
    d, w = _model(key, seed)
    return ORACLES[d["architecture"]].forward(d, w, list(toks), torch.float64).float()


def want_logits(d, toks, seed=0):
    return _oracle(json.dumps(d), seed, tuple(toks))


def session(d, dtype, blocks=64, slots=4, seed=0, block_size=16, weights=None):
    from art_b200.engine.factory import build_runner
    from art_b200.engine.kv_cache import BlockManager
    from art_b200.engine.replay import Replay
    from art_b200.models.config import config_from_dict

    cfg = config_from_dict(d)
    runner, kv = build_runner(cfg, weights or model(d, seed)[1], num_blocks=blocks, block_size=block_size, num_slots=slots, dtype=dtype)
    return Replay(runner, BlockManager(blocks, block_size, False), kv)


def feed(rep, toks, cuts, name="a"):
    """Logits of every position, the tokens cut into portions of the given sizes (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        last = at + n == len(toks)
        out.append(rep.step([{"id": name, "tokens": toks[at:at + n], "want": list(range(n))}], [name] if last else []).cpu())
        at, i = at + n, i + 1
    return torch.cat(out)


def errors(got, want):
    assert torch.isfinite(got).all()
    return (got.float() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def check(got, want, dtype, scale=1.0):
    err = errors(got, want)
    assert float(err.max()) < TOL[dtype] * scale, f"worst {float(err.max()):.2e} at {int(err.argmax())}"


def check_routed(got, want, dtype, scale=1.0):
    """As ``check``, for models with a router: in bf16 rounding moves a close call to another expert now and then."""
    if dtype == F32:
        return check(got, want, dtype, scale)
    err = errors(got, want)
    over = (err >= TOL[dtype] * scale).float().mean()
    assert float(over) <= 0.06 and float(err.max()) < 0.8, f"{float(over):.3f} of the positions are off, worst {float(err.max()):.2e} at {int(err.argmax())}"


def mixed_session(d, dtype, lens, compare, blocks=40, seed=4):
    """Portions beside single tokens, requests that pause, end and make room for others; each as if it ran alone."""
    n_req = len(lens)
    reqs = [tokens(n, d["vocab"], 10 + i) for i, n in enumerate(lens)]
    rep = session(d, dtype, blocks=blocks, slots=4)
    g = torch.Generator().manual_seed(seed)
    at, got, live, nxt = [0] * n_req, [[] for _ in lens], [], 0
    while nxt < n_req or live:
        held = sum((lens[i] + 15) // 16 for i in live)
        while nxt < n_req and len(live) < 4 and held + (lens[nxt] + 15) // 16 <= blocks:
            held += (lens[nxt] + 15) // 16
            live.append(nxt)
            nxt += 1
        act = [i for i in live if torch.rand(1, generator=g).item() < 0.8] or live[:1]
        entries, end, rows = [], [], []
        for i in act:
            n = min([1, 1, 2, 19, 64, 100][int(torch.randint(0, 6, (1,), generator=g))], lens[i] - at[i])
            entries.append({"id": str(i), "tokens": reqs[i][at[i]:at[i] + n], "want": list(range(n))})
            rows.append((i, n))
            at[i] += n
            if at[i] == lens[i]:
                end.append(str(i))
        out = rep.step(entries, end).cpu()
        for i, n in rows:
            got[i].append(out[:n])
            out = out[n:]
        live = [i for i in live if at[i] < lens[i]]
    assert rep.bm.num_free == blocks and (rep.state_slots is None or rep.state_slots.num_free == 4)
    for i, r in enumerate(reqs):
        compare(torch.cat(got[i]), want_logits(d, r), dtype, 1.5)
