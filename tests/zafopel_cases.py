"""Small random Zafopel models for the tests: configurations with unlike layers, and checkpoint tensors for them."""
from __future__ import annotations

import math

import torch


def layer(heads, dim, rot, vdim, rank, scale, base, window=None, q_rank=None, kv_from=None, mlp=None):
    """``q_rank``: queries through a latent, causal, with a sink; without it: straight queries and a sliding window."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if window:
        m["mask"] = {"size": window}
    if q_rank:
        m["q_rank"] = q_rank
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention_2" if q_rank else "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Zafopel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def unlike():
    """Every layer its own sizes, none a multiple of 8 where it need not be: layers that read an earlier layer's latents (with a longer window
    than that layer's own, and without a window), more heads than a tile, one expert, no feed-forward."""
    return config(100, 301, [
        layer(5, 20, 12, 28, 36, 0.3, 5000.0, q_rank=44, mlp=moe(6, 3, 36)),
        layer(3, 24, 6, 16, 42, 0.25, 700.0, window=37, mlp=dense(50)),
        layer(7, 40, 6, 24, 42, 0.2, 700.0, window=100, kv_from=1, mlp=moe(5, 1, 20)),
        layer(2, 16, 12, 10, 36, 0.4, 5000.0, q_rank=21, kv_from=0),
        layer(40, 8, 2, 8, 136, 0.5, 60.0, window=64, mlp=moe(1, 1, 24)),
    ])


def sliding():
    """Windows everywhere (no multiples of a page), so old pages go back while a request runs."""
    return config(128, 256, [
        layer(8, 64, 32, 64, 128, 0.12, 10000.0, window=90, mlp=moe(8, 2, 64)),
        layer(4, 48, 32, 40, 128, 0.15, 10000.0, window=70, kv_from=0, mlp=dense(248)),
        layer(8, 64, 32, 64, 128, 0.12, 10000.0, window=90, mlp=moe(8, 2, 64)),
    ], 1e-6)


def wide():
    """Latents and heads of full size, two tiles of heads, a short and a page-sized window; and a latent only the CUDA cores take."""
    return config(64, 128, [
        layer(33, 128, 64, 128, 512, 0.08, 10000.0, q_rank=72, mlp=dense(64)),
        layer(2, 128, 64, 96, 320, 0.08, 10000.0, window=200, mlp=moe(4, 2, 32)),
        layer(3, 32, 16, 32, 600, 0.2, 10000.0, window=5),
        layer(6, 160, 40, 144, 64, 0.1, 10000.0, window=64, mlp=dense(40)),
    ], 1e-6)


def tensors(cfg, seed=0):
    """bf16 checkpoint tensors whose outputs keep unit scale and whose scores spread over several units."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape):
        return torch.randn(*shape, generator=g)

    def lin(rows, cols, gain=1.0):
        return gain * rnd(rows, cols) / math.sqrt(cols)

    d = cfg["width"]
    t = {"embed": rnd(cfg["vocab"], d), "head": lin(cfg["vocab"], d)}

    def norm(name, alpha):
        t[name], t[name + ".b"], t[name + ".alpha"] = 1 + 0.3 * rnd(d), 0.3 * rnd(d), torch.tensor(alpha)

    norm("final.norm", 0.4)
    for i, l in enumerate(cfg["layers"]):
        m, e = l["mixer"], l["mlp"]
        h, q_rows = m["heads"], m["heads"] * (m["dim"] + m["rot_dim"])
        p = f"l{i}.mix."
        norm(f"l{i}.norm1", 0.9 - 0.1 * i)
        if "q_rank" in m:
            t[p + "dq"], t[p + "dq.norm"] = lin(m["q_rank"], d), 1 + 0.3 * rnd(m["q_rank"])
            t[p + "uq"], t[p + "sink"] = lin(q_rows, m["q_rank"], 2.0), 1 + 2 * rnd(h)
        else:
            t[p + "q"] = lin(q_rows, d, 2.0)
        if "kv_from" not in m:
            t[p + "dkv"], t[p + "dkv.norm"] = lin(m["kv_rank"] + m["rot_dim"], d), 1 + 0.3 * rnd(m["kv_rank"])
        t[p + "uk"], t[p + "uv"] = lin(h * m["dim"], m["kv_rank"]), lin(h * m["vdim"], m["kv_rank"])
        t[p + "o"] = lin(d, h * m["vdim"])
        p = f"l{i}.mlp."
        if e is None:
            continue
        if e["kind"] == "dense":
            t[p + "up"], t[p + "down"] = lin(e["ff"], d), lin(d, e["ff"])
            continue
        f = e["expert"]["ff"]
        t[p + "router"] = lin(e["router"]["experts"], d, 2.0)
        for s in range(e["router"]["experts"]):
            t[p + f"e{s}.gate"], t[p + f"e{s}.up"], t[p + f"e{s}.down"] = lin(f, d, 2.0), lin(f, d, 2.0), lin(d, f)
    return {n: v.bfloat16() for n, v in t.items()}
