"""Plain, slow restatement of the Gaparax equations: the oracle of that design's tests.

One function per mechanism, ordinary PyTorch on the CPU, no cache, no batching, whole sequences at a time.  Nothing here is
shared with the product path.  ``dtype`` of the weights decides the precision (the tests use float64).
"""
import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def relu2(z):
    return z.clamp(min=0) ** 2


def silu(z):
    return z * sigmoid(z)


def part(w, name):
    return {k[len(name) + 1:]: t for k, t in w.items() if k.startswith(name + ".")}


def bucket(n, rows, reach):
    """Row of the distance table: one per distance for the near half, then logarithmic up to ``reach``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def distance_bias(T, table, reach):
    """[T, T, H]: what the score of query i and key j gains; entries with j > i are not used."""
    out = torch.zeros(T, T, table.shape[1], dtype=table.dtype)
    rows = torch.tensor([bucket(n, table.shape[0], reach) for n in range(T)])
    for i in range(T):
        out[i, :i + 1] = table[rows[:i + 1].flip(0)]
    return out


def chunk_mask(T, size):
    """[T, T]: True where query i sees key j."""
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def attention(h, w, p, eps):
    """Weights are sigmoids of the scores of a query's own chunk; nothing is divided by their sum."""
    T, H, G = h.shape[0], p["heads"], p["kv_heads"]
    q = rms((h @ w["q"].T).view(T, H, p["dim"]), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).view(T, G, p["dim"]), eps) * w["k.norm"]
    v = (h @ w["v"].T).view(T, G, p["vdim"])
    bias, seen = distance_bias(T, w["rel"], p["bias_max"]), chunk_mask(T, p["mask"]["size"])
    out = torch.zeros(T, H, p["vdim"], dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        s = q[:, n] @ k[:, g].T * p["scale"] * w["temp"][n]
        s = p["softcap"] * torch.tanh(s / p["softcap"]) if p["softcap"] else s
        out[:, n] = (sigmoid(s + bias[:, :, n] + w["pb"][n]) * seen) @ v[:, g]
    return (out.reshape(T, -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


def frequencies(rot):
    """(one frequency per pair, factor of sine and cosine): geometric, or blended with their interpolation where the turns
    a pair makes over the original context say so."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if s is None:
        return f, 1.0

    def pair_of(turns):
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot):
    """x [T, heads, dims]: dimension i turns with dimension i + dims / 2."""
    f, m = frequencies(rot)
    out, half = x.clone(), rot["dims"] // 2
    for i in range(half):
        ang = torch.arange(x.shape[0], dtype=torch.float64) * f[i]
        c, s = (m * torch.cos(ang)).to(x.dtype)[:, None], (m * torch.sin(ang)).to(x.dtype)[:, None]
        out[..., i] = x[..., i] * c - x[..., i + half] * s
        out[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return out


def sink_softmax(s, sink):
    """Softmax of a row of scores whose denominator has one more term, exp(sink)."""
    m = torch.maximum(s.amax(-1, keepdim=True), sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def latent_attention(h, w, p, eps):
    T, H, dim, rot, rank = h.shape[0], p["heads"], p["dim"], p["rot_dim"], p["kv_rank"]
    q = (h @ w["q"].T).view(T, H, dim + rot)
    down = h @ w["dkv"].T
    c = rms(down[:, :rank], eps) * w["dkv.norm"]
    kr = rotate(down[:, None, rank:], p["rot"])[:, 0]
    qr = rotate(q[..., dim:], p["rot"])
    k, v = (c @ w["uk"].T).view(T, H, dim), (c @ w["uv"].T).view(T, H, p["vdim"])
    hidden = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    out = torch.zeros(T, H, p["vdim"], dtype=h.dtype)
    for n in range(H):
        s = (q[:, n, :dim] @ k[:, n].T + qr[:, n] @ kr.T) * p["scale"]
        out[:, n] = sink_softmax(s.masked_fill(hidden, -math.inf), w["sink"][n]) @ v[:, n]
    return out.reshape(T, -1) @ w["o"].T


def dense(h, w):
    return relu2(h @ w["up"].T) @ w["down"].T


def expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, w, r):
    """Chosen experts and their weights, [T, top] each: only the best groups' experts can be chosen."""
    s = torch.softmax(h @ w["router"].T, -1)
    T, E = s.shape
    n = r["groups"]["count"]
    best = s.view(T, n, E // n).amax(-1).sort(dim=-1, descending=True, stable=True).indices[:, :r["groups"]["keep"]]
    kept = torch.zeros(T, n, dtype=torch.bool).scatter(1, best, True).repeat_interleave(E // n, 1)
    top = s.masked_fill(~kept, -1.0).sort(dim=-1, descending=True, stable=True).indices[:, :r["top"]]
    return top, s.gather(-1, top) * r["scale"]


def moe(h, w, p):
    best, a = route(h, w, p["router"])
    out = torch.zeros_like(h)
    for e in range(p["router"]["experts"]):
        for s in range(best.shape[1]):
            rows = best[:, s] == e
            if rows.any():
                out[rows] += a[rows, s, None] * expert(h[rows], part(w, f"e{e}"))
    return out


def boundary(xs, w, k, norm, eps, sublayer):
    """Hyper-connected streams xs [S, T, d] across sublayer ``k``, whose result passes a gate of its input."""
    hc = part(w, f"hc{k}")
    u = sum(a * x for a, x in zip(hc["in"], xs))
    h = rms(u, eps) * norm
    y = sublayer(h) * sigmoid(h @ w[f"rg{k}"].T + w[f"rg{k}.b"])
    return torch.stack([sum(hc["mix"][s, t] * xs[s] for s in range(len(xs))) + hc["out"][t] * y for t in range(len(xs))])


MIXERS = {"attention": attention, "latent_attention": latent_attention}


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: list that receives the sum of the streams after every layer."""
    W = {k: t.to(dtype) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    xs = W["embed"][torch.as_tensor(tokens)].expand(cfg["streams"], -1, -1)
    for i, layer in enumerate(cfg["layers"]):
        w = part(W, f"l{i}")
        xs = boundary(xs, w, 1, w["norm1"], eps, lambda h: MIXERS[layer["type"]](h, part(w, "mix"), layer["mixer"], eps))
        if layer["mlp"] is not None:
            m = part(w, "mlp")
            xs = boundary(xs, w, 2, w["norm2"], eps, lambda h: dense(h, m) if layer["mlp"]["kind"] == "dense" else moe(h, m, layer["mlp"]))
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return (rms(xs.sum(0), eps) * W["final.norm"]) @ W["head"].T
