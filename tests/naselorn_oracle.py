"""Plain, slow restatement of the Naselorn equations: the oracle of that design's tests.

One function per mechanism, ordinary PyTorch on the CPU, no cache, no batching, loops over tokens where the mechanism is
a recurrence.  Nothing here is shared with the product path.  ``dtype`` of the weights decides the precision (the tests
use float64).
"""
import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def sinusoids(n, width, dtype=torch.float64):
    """Position vectors of positions 0 .. n - 1: sine at even entries, cosine of the same angle at odd ones."""
    out = torch.zeros(n, width, dtype=torch.float64)
    for c in range(width):
        ang = torch.arange(n, dtype=torch.float64) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.cos(ang) if c % 2 else torch.sin(ang)
    return out.to(dtype)


def chunked_attention(h, w, p):
    """Grouped-query attention without rotation; a token sees its own chunk of the sequence up to itself."""
    T = h.shape[0]
    H, G, dim, vdim = p["heads"], p["heads"] // p["kv_heads"], p["dim"], p["vdim"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, dim)
    k = (h @ w["k"].T + w["k.b"]).view(T, -1, dim)
    v = (h @ w["v"].T + w["v.b"]).view(T, -1, vdim)
    C = p["mask"]["size"]
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for i in range(T):
        lo = i // C * C
        for n in range(H):
            a = torch.softmax(k[lo:i + 1, n // G] @ q[i, n] * p["scale"], -1)
            out[i, n] = a @ v[lo:i + 1, n // G]
    return out.reshape(T, H * vdim) @ w["o"].T + w["o.b"]


def short_conv(x, taps, bias):
    """Causal convolution per channel; the last tap meets the current token."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            if t - (n - 1) + j >= 0:
                out[t] += taps[:, j] * x[t - (n - 1) + j]
    return out + bias


def rglru(h, w, p):
    """Gated recurrence per channel behind a short convolution, times a gelu branch."""
    T, n, blocks = h.shape[0], p["width"], p["blocks"]
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = short_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    ub = u.view(T, blocks, n // blocks)
    r, i = torch.zeros_like(ub), torch.zeros_like(ub)
    for b in range(blocks):
        r[:, b] = sigmoid(ub[:, b] @ w["ra"][b].T + w["ra.b"][b])
        i[:, b] = sigmoid(ub[:, b] @ w["ri"][b].T + w["ri.b"][b])
    r, i = r.reshape(T, n), i.reshape(T, n)
    S, out = torch.zeros(n, dtype=h.dtype), torch.zeros_like(u)
    for t in range(T):
        log_a = -8 * r[t] * softplus(w["lam"])
        a = torch.exp(log_a)
        S = a * S + torch.sqrt(1 - a * a) * i[t] * u[t]
        out[t] = S
    return (out * y) @ w["o"].T


def part(w, name):
    return {k[len(name) + 1:]: t for k, t in w.items() if k.startswith(name + ".")}


def parallel(h, w, p, eps):
    return p["left_scale"] * chunked_attention(h, part(w, "left"), p["left"]) + p["right_scale"] * rglru(h, part(w, "right"), p["right"])


def lightning(h, w, p, eps):
    T, H, dim, vdim = h.shape[0], p["heads"], p["dim"], p["vdim"]
    q, k = (silu(h @ w[n].T).view(T, H, dim) for n in "qk")
    v = silu(h @ w["v"].T).view(T, H, vdim)
    decay = torch.tensor(p["decay"], dtype=h.dtype).view(H, 1, 1)
    S = torch.zeros(H, dim, vdim, dtype=h.dtype)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for t in range(T):
        S = decay * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    o = rms(out.reshape(T, H * vdim), eps) * w["norm"] * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def gated(h, w, act):
    return (act(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def moe(h, w, p):
    z = h @ w["router"].T + w["router.b"]
    out = gated(h, part(w, "shared"), silu) if p.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        best = sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[:p["router"]["top"]]
        a = torch.softmax(z[t, best], -1)
        for c, e in zip(a, best):
            out[t] = out[t] + c * gated(h[t:t + 1], part(w, f"e{e}"), silu)[0]
    return out


MIXERS = {"parallel": parallel, "lightning": lightning}


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: list that receives the residual stream after every layer."""
    W = {k: t.to(dtype) for k, t in weights.items()}
    eps, width = cfg["norm"]["eps"], cfg["width"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"] + sinusoids(len(tokens), width, dtype)
    for i, layer in enumerate(cfg["layers"]):
        w = part(W, f"l{i}")
        x = x + MIXERS[layer["type"]](rms(x, eps) * (1 + w["norm1"]), part(w, "mix"), layer["mixer"], eps)
        p = layer["mlp"]
        if p is not None:
            h, m = rms(x, eps) * (1 + w["norm2"]), part(w, "mlp")
            x = x + (gated(h, m, lambda z: z.clamp(min=0)) if p["kind"] == "dense" else moe(h, m, p))
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * (1 + W["final.norm"])) @ W["head"].T
