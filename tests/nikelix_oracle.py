"""Plain, slow restatement of the Nikelix equations: the oracle of the hybrid-model tests.

One function per mechanism, ordinary PyTorch on the CPU, no cache, no batching, loops over tokens where the
mechanism is a recurrence.  Nothing here is shared with the product path.  ``dtype`` of the weights decides the
precision (the tests use float64 or float32).
"""
import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def rotate_pairs(x, positions, base):
    """Interleaved rotary embedding of every element of the last axis: the pair (2i, 2i+1) turns by p * base^(-2i/n)."""
    n = x.shape[-1]
    out = x.clone()
    for i in range(n // 2):
        ang = positions.to(torch.float64) * float(base) ** (-2.0 * i / n)
        c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
        while c.dim() < x.dim() - 1:
            c, s = c.unsqueeze(-1), s.unsqueeze(-1)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def latent_attention(h, w, p, eps):
    """h [T, d]; w: name -> tensor; p: the mixer's sizes and constants."""
    T = h.shape[0]
    H, dim, rot, vdim, rank = p["heads"], p["dim"], p["rot_dim"], p["vdim"], p["kv_rank"]
    q = (h @ w["q"].T).view(T, H, dim + rot)
    low = h @ w["dkv"].T
    c = rms(low[:, :rank], eps) * w["dkv.norm"]
    pos = torch.arange(T)
    k_rot = rotate_pairs(low[:, rank:], pos, p["rot"]["base"])
    q_rot = rotate_pairs(q[..., dim:], pos, p["rot"]["base"])
    k = (c @ w["uk"].T).view(T, H, dim)
    v = (c @ w["uv"].T).view(T, H, vdim)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    window = p["mask"]["size"]
    for i in range(T):
        lo = max(0, i - window + 1)
        s = torch.einsum("hd,jhd->hj", q[i, :, :dim], k[lo:i + 1]) + q_rot[i] @ k_rot[lo:i + 1].T
        a = torch.softmax(s * p["scale"], -1)
        out[i] = torch.einsum("hj,jhd->hd", a, v[lo:i + 1])
    return out.reshape(T, H * vdim) @ w["o"].T


def hgrn2(h, w, p, eps):
    T = h.shape[0]
    H, dim, vdim = p["heads"], p["dim"], p["vdim"]
    q = silu(h @ w["q"].T).view(T, H, dim)
    v = (h @ w["v"].T).view(T, H, vdim)
    low = w["lower"].view(H, dim)
    f = low + (1 - low) * torch.sigmoid(h @ w["f"].T + w["f.b"]).view(T, H, dim)
    S = torch.zeros(H, dim, vdim, dtype=h.dtype)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for t in range(T):
        S = f[t].unsqueeze(-1) * S + (1 - f[t]).unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    out = rms(out, eps) * w["norm"]
    return out.reshape(T, H * vdim) @ w["o"].T


def wkv(h, w, p, eps):
    T = h.shape[0]
    H, dim = p["heads"], p["dim"]
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    mix = {s: h + (prev - h) * w["mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[s].T).view(T, H, dim) for s in "rkv")
    gate = silu(mix["g"] @ w["g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).view(T, H, dim)
    u = w["u"].view(H, dim)
    S = torch.zeros(H, dim, dim, dtype=h.dtype)
    out = torch.zeros(T, H, dim, dtype=h.dtype)
    for t in range(T):
        kv = k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hkv,hk->hv", S + u.unsqueeze(-1) * kv, r[t])
        S = decay[t].unsqueeze(-1) * S + kv
    out = rms(out, eps).reshape(T, H * dim) * w["norm"] * gate
    return out @ w["o"].T


def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


MIXERS = {"latent_attention": latent_attention, "hgrn2": hgrn2, "wkv": wkv}


def forward(cfg, weights, tokens, dtype=torch.float32, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: list that receives the residual stream after every layer."""
    W = {k: t.to(dtype) for k, t in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = rms(W["embed"][torch.as_tensor(tokens)], eps) * W["embed.norm"]
    hist = [x]
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        mix = {k[len(pre) + 4:]: t for k, t in W.items() if k.startswith(pre + "mix.")}
        y = MIXERS[layer["type"]](rms(x, eps) * W[pre + "norm1"], mix, layer["mixer"], eps)
        x = x + m * rms(y, eps) * W[pre + "norm1b"]
        if layer["mlp"] is not None:
            z = (rms(x, eps) * W[pre + "norm2"]) @ W[pre + "mlp.up"].T
            y = poly_norm(z, W[pre + "mlp.act"], eps) @ W[pre + "mlp.down"].T
            x = x + m * rms(y, eps) * W[pre + "norm2b"]
        hist.append(x)
        x = sum(W[pre + "dwa"][j] * hist[j] for j in range(i + 2))
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["embed"].T
