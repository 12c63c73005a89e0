"""Plain, slow restatement of the Dulisun decoder, one function per mechanism (float64 on the CPU).

Shares no code with the package: it takes the ``config.json`` dictionary and a dictionary of tensors under their
checkpoint names. ``forward`` runs whole sequences only; caches, portions and batches are the product's business."""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """RMS norm whose weight is stored as the difference from one."""
    return rms(x, eps) * (1.0 + w)


def rotate(x, positions, base, dims):
    """Interleaved rotary embedding of the first ``dims`` entries of the last axis; x is [tokens, heads, dim]."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(n, size):
    """[n, n] mask: position i sees j <= i of its own chunk of ``size`` positions (None: every j <= i)."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    m = j <= i
    return m if size is None else m & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def attend(q, k, v, mask, scale, sink):
    """Softmax attention, q [n, H, dim], k [m, G, dim], v [m, G, vdim]; exp(sink[h]) joins the denominator of head h."""
    n, heads, _ = q.shape
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for h in range(heads):
        g = h // (heads // k.shape[1])
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(~mask, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[h].expand(n, 1)], 1)
        p = torch.softmax(s, -1)[:, : k.shape[0]]
        out[:, h] = p @ v[:, g]
    return out


def attention(h, t, pre, m, eps):
    n = h.shape[0]
    heads, kv, dim = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ t[pre + "q"].T).view(n, heads, dim)
    k = (h @ t[pre + "k"].T).view(n, kv, dim)
    v = k
    pos = torch.arange(n)
    rot = m.get("rot")
    if rot:
        q, k = rotate(q, pos, rot["base"], rot["dims"]), rotate(k, pos, rot["base"], rot["dims"])
    q, k = rms(q, eps), rms(k, eps)
    mask = m.get("mask")
    o = attend(q, k, v, visible(n, mask["size"] if mask else None), m["scale"], t[pre + "sink"])
    return o.reshape(n, heads * dim) @ t[pre + "o"].T


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def ffn(h, t, pre):
    return gelu(h @ t[pre + "up"].T) @ t[pre + "down"].T


def route(scores, router):
    """Chosen expert numbers (best first) for one token's scores."""
    n, groups = router["experts"], router.get("groups") or {"count": 1, "keep": 1}
    per = n // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -max(scores[g * per:(g + 1) * per]))[: groups["keep"]]
    allowed = [e for e in range(n) if e // per in best]
    return sorted(allowed, key=lambda e: -scores[e])[: router["top"]]


def moe(h, t, pre, m):
    out = torch.zeros_like(h)
    s = torch.softmax(h @ t[pre + "router"].T, -1)
    for i in range(h.shape[0]):
        for e in route(s[i].tolist(), m["router"]):
            out[i] += s[i, e] * ffn(h[i:i + 1], t, f"{pre}e{e}.")[0]
    if m.get("shared"):
        out += ffn(h, t, pre + "shared.")
    return out


def forward(config, tensors, tokens, layers_out=None):
    """Logits [tokens, vocab]; ``layers_out`` (a list) receives the residual stream after every layer."""
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = norm(t["embed"][torch.as_tensor(tokens, dtype=torch.long)], t["embed.norm"], eps)
    for i, layer in enumerate(config["layers"]):
        x = x + norm(attention(x, t, f"l{i}.mix.", layer["mixer"], eps), t[f"l{i}.norm1"], eps)
        if layer["mlp"] is not None:
            x = x + norm(moe(x, t, f"l{i}.mlp.", layer["mlp"]), t[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, t["final.norm"], eps) @ t["embed"].T
