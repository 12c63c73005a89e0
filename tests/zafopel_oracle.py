"""Plain, slow restatement of the Zafopel decoder, one function per mechanism (float64 on the CPU).

Shares no code with the package: it takes the ``config.json`` dictionary and a dictionary of tensors under their
checkpoint names. ``forward`` runs whole sequences only; caches, portions and batches are the product's business."""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def dynamic_tanh(x, t, name):
    """Elementwise bounded norm: no statistics of x enter it."""
    return torch.tanh(t[name + ".alpha"] * x) * t[name] + t[name + ".b"]


def rms(x, w, eps):
    """x over its root mean square along the last axis (eps inside the root), times the plain weight."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate(x, positions, base):
    """Interleaved rotary embedding of the whole last axis; x is [tokens, ..., dims]."""
    dims = x.shape[-1]
    out = x.clone()
    shape = (-1,) + (1,) * (x.dim() - 2)
    for i in range(dims // 2):
        a = (positions.to(F64) * base ** (-2.0 * i / dims)).view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def visible(n, size):
    """[n, n] mask: position i sees itself and the ``size - 1`` positions before it (None: every j <= i)."""
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) if size is None else (back >= 0) & (back < size)


def attend(q, k, v, mask, scale, sink):
    """Softmax attention head by head, q and k [n, H, d], v [n, H, vd]; exp(sink[h]) joins the denominator of head h."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[-1], dtype=q.dtype)
    for h in range(q.shape[1]):
        s = ((q[:, h] @ k[:, h].T) * scale).masked_fill(~mask, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[h].expand(s.shape[0], 1)], 1)
        out[:, h] = torch.softmax(s, -1)[:, : k.shape[0]] @ v[:, h]
    return out


def latent(h, t, pre, m, eps):
    """What a layer's cache holds per token: the normed latent and the rotated key part all heads share."""
    both = h @ t[pre + "dkv"].T
    r = m["kv_rank"]
    return rms(both[:, :r], t[pre + "dkv.norm"], eps), rotate(both[:, r:], torch.arange(h.shape[0]), m["rot"]["base"])


def queries(h, t, pre, m, eps, through_latent):
    """Per head [dim unrotated, rot_dim rotated]."""
    q = rms(h @ t[pre + "dq"].T, t[pre + "dq.norm"], eps) @ t[pre + "uq"].T if through_latent else h @ t[pre + "q"].T
    q = q.view(h.shape[0], m["heads"], m["dim"] + m["rot_dim"])
    return torch.cat([q[..., : m["dim"]], rotate(q[..., m["dim"]:], torch.arange(h.shape[0]), m["rot"]["base"])], -1)


def mixer(h, t, pre, layer, eps, latents):
    """``latents`` holds every earlier layer's cached pair; a layer with ``kv_from`` takes one of them instead of its own."""
    m, n = layer["mixer"], h.shape[0]
    second = layer["type"] == "latent_attention_2"
    c, k_rot = latents[m["kv_from"]] if "kv_from" in m else latent(h, t, pre, m, eps)
    latents.append((c, k_rot))
    q = queries(h, t, pre, m, eps, second)
    k = (c @ t[pre + "uk"].T).view(n, m["heads"], m["dim"])
    v = (c @ t[pre + "uv"].T).view(n, m["heads"], m["vdim"])
    k = torch.cat([k, k_rot[:, None].expand(n, m["heads"], m["rot_dim"])], -1)
    mask = visible(n, None if second else m["mask"]["size"])
    o = attend(q, k, v, mask, m["scale"], t[pre + "sink"] if second else None)
    return o.reshape(n, -1) @ t[pre + "o"].T


def dense(h, t, pre):
    return torch.relu(h @ t[pre + "up"].T) ** 2 @ t[pre + "down"].T


def expert(h, t, pre):
    z = h @ t[pre + "gate"].T
    return (z * torch.sigmoid(z) * (h @ t[pre + "up"].T)) @ t[pre + "down"].T


def route(h, t, pre, router):
    """(scores of every expert, chosen expert numbers best first) for the rows of h."""
    s = torch.sigmoid(h @ t[pre + "router"].T)
    return s, [sorted(range(router["experts"]), key=lambda e: -row[e])[: router["top"]] for row in s.tolist()]


def moe(h, t, pre, m):
    out = torch.zeros_like(h)
    s, chosen = route(h, t, pre, m["router"])
    for i, row in enumerate(chosen):
        for e in row:
            out[i] += expert(s[i, e] * h[i:i + 1], t, f"{pre}e{e}.")[0]
    return out


def forward(config, tensors, tokens, layers_out=None):
    """Logits [tokens, vocab]; ``layers_out`` (a list) receives the residual stream after every layer."""
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    latents = []
    for i, layer in enumerate(config["layers"]):
        h = dynamic_tanh(x, t, f"l{i}.norm1")
        add = mixer(h, t, f"l{i}.mix.", layer, eps, latents)
        if layer["mlp"] is not None:
            add = add + (moe(h, t, f"l{i}.mlp.", layer["mlp"]) if layer["mlp"]["kind"] == "moe" else dense(h, t, f"l{i}.mlp."))
        x = x + add
        if layers_out is not None:
            layers_out.append(x)
    return dynamic_tanh(x, t, "final.norm") @ t["head"].T
