"""Plain, slow restatement of the Gaborax equations: the oracle of that design's tests.

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


def part(w, name):
    return {k[len(name) + 1:]: t for k, t in w.items() if k.startswith(name + ".")}


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


def rotate(x, rot, interleaved):
    """x [T, heads, dim]: the first ``dims`` dimensions of every head turn by their position's angles."""
    f, m = frequencies(rot)
    out = x.clone()
    n = rot["dims"]
    for i in range(n // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n // 2)
        ang = torch.arange(x.shape[0], dtype=torch.float64) * f[i]
        c, s = (m * torch.cos(ang)).to(x.dtype)[:, None], (m * torch.sin(ang)).to(x.dtype)[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def keys_values(h, w, p, eps, interleaved):
    T, bias = h.shape[0], interleaved
    k, v = h @ w["k"].T, h @ w["v"].T
    if bias:
        k, v = k + w["k.b"], v + w["v.b"]
    k = (rms(k, eps) * w["k.norm"]).view(T, p["kv_heads"], p["dim"])
    return rotate(k, p["rot"], interleaved), v.view(T, p["kv_heads"], p["vdim"])


def attend(q, k, v, scale, softcap=None):
    """Causal softmax attention, q [T, H, dim], k and v [T, G, .]; scores may be squashed into (-softcap, softcap)."""
    T, H = q.shape[:2]
    g = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    hidden = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    for n in range(H):
        s = q[:, n] @ k[:, n // g].T * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        out[:, n] = torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, n // g]
    return out


def attention(h, w, p, eps, kv):
    """Rotate-half attention with a gate per head.  ``kv``: keys and values of the layer itself or of the one it shares with."""
    T, H = h.shape[0], p["heads"]
    q = rotate((rms(h @ w["q"].T, eps) * w["q.norm"]).view(T, H, p["dim"]), p["rot"], False)
    o = attend(q, *kv, p["scale"]) * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, -1) @ w["o"].T


def attention_2(h, w, p, eps, kv):
    """Interleaved rotation, biases, squashed scores."""
    T, H = h.shape[0], p["heads"]
    q = rotate((rms(h @ w["q"].T + w["q.b"], eps) * w["q.norm"]).view(T, H, p["dim"]), p["rot"], True)
    return attend(q, *kv, p["scale"], p["softcap"]).reshape(T, -1) @ w["o"].T


def expert(h, w):
    return relu2(h @ w["up"].T) @ w["down"].T


def route(h, w, p):
    """Chosen outputs and their weights, [T, top] each.  Outputs past the real experts hand the input on."""
    s = torch.softmax(h @ w["router"].T, -1)
    best = (s + w["correction"]).sort(dim=-1, descending=True, stable=True).indices[:, :p["router"]["top"]]
    a = s.gather(-1, best)
    return best, a / (a.sum(-1, keepdim=True) + 1e-20)


def moe(h, w, p):
    out = sigmoid(h @ w["shared.sg"].T) * expert(h, part(w, "shared")) if p.get("shared") else torch.zeros_like(h)
    best, a = route(h, w, p)
    n = p["router"]["experts"]
    for e in range(n + p["router"].get("identity", 0)):
        for s in range(best.shape[1]):
            rows = best[:, s] == e
            if rows.any():
                out[rows] += a[rows, s, None] * (expert(h[rows], part(w, f"e{e}")) if e < n else h[rows])
    return out


MIXERS = {"attention": (attention, False), "attention_2": (attention_2, True)}


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: list that receives the residual stream after every layer."""
    W = {k: t.to(dtype) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        w, p = part(W, f"l{i}"), layer["mixer"]
        fn, interleaved = MIXERS[layer["type"]]
        m = part(w, "mix")
        kept[i] = kept[p["kv_from"]] if "kv_from" in p else keys_values(x, m, p, eps, interleaved)
        x = x + rms(fn(x, m, p, eps, kept[i]), eps) * (1 + w["norm1"]) * w["ls1"]
        if layer["mlp"] is not None:
            x = x + rms(moe(x, part(w, "mlp"), layer["mlp"]), eps) * (1 + w["norm2"]) * w["ls2"]
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * (1 + W["final.norm"])) @ W["embed"].T
