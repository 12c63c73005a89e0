"""Small random Dulisun models for the tests: configurations with unlike layers, and checkpoints written to a directory."""
from __future__ import annotations

import json
import math

import torch


def layer(heads, kv, dim, scale, window=None, rot=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def moe(experts, top, ff, groups=None, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Dulisun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def unlike():
    """Every layer its own sizes: odd widths, one head per group and many, no rotation, no chunks, a head wider than the
    tensor-core prompt kernel takes, one expert, a shared part that is no multiple of the experts, a layer without feed-forward."""
    return config(100, 301, [
        layer(6, 3, 20, 0.3, 50, (5000.0, 12), moe(6, 3, 36, (3, 2), 50)),
        layer(10, 1, 40, 0.2, 130, (10000.0, 40)),
        layer(4, 4, 136, 0.09, None, None, moe(5, 1, 64)),
        layer(2, 2, 64, 0.15, 64, (700.0, 2), moe(1, 1, 24, (1, 1), 8)),
    ])


def regular():
    """Equal layers, a multiple of 8 everywhere, chunks that are no multiple of a page."""
    return config(128, 256, [layer(8, 2, 48, 0.25, 90, (10000.0, 32), moe(8, 2, 64, (4, 2), 128)) for _ in range(2)], 1e-6)


def long_chunks():
    """Chunks of several pages and of several key tiles."""
    return config(64, 128, [layer(4, 1, 32, 0.3, w, (10000.0, 16), moe(4, 2, 32, (2, 1), 32)) for w in (200, 320)], 1e-6)


def tensors(cfg, seed=0, sink_shift=0.0):
    """bf16 checkpoint tensors whose outputs keep unit scale and whose scores spread over several units."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape):
        return torch.randn(*shape, generator=g)

    d = cfg["width"]
    t = {"embed": rnd(cfg["vocab"], d) / math.sqrt(d), "embed.norm": 0.3 * rnd(d), "final.norm": 0.3 * rnd(d)}
    for i, l in enumerate(cfg["layers"]):
        m = l["mixer"]
        h, k, hd = m["heads"], m["kv_heads"], m["dim"]
        p = f"l{i}."
        t[p + "norm1"] = 0.3 * rnd(d)
        t[p + "mix.q"], t[p + "mix.k"] = rnd(h * hd, d) / math.sqrt(d), rnd(k * hd, d) / math.sqrt(d)
        t[p + "mix.o"], t[p + "mix.sink"] = rnd(d, h * hd) / math.sqrt(h * hd), rnd(h) + sink_shift
        if l["mlp"] is not None:
            e = l["mlp"]
            f = e["expert"]["ff"]
            t[p + "norm2"] = 0.3 * rnd(d)
            t[p + "mlp.router"] = 2.0 * rnd(e["router"]["experts"], d) / math.sqrt(d)
            for s in range(e["router"]["experts"]):
                t[p + f"mlp.e{s}.up"], t[p + f"mlp.e{s}.down"] = rnd(f, d) / math.sqrt(d), rnd(d, f) / math.sqrt(f)
            if e.get("shared"):
                fs = e["shared"]["ff"]
                t[p + "mlp.shared.up"], t[p + "mlp.shared.down"] = rnd(fs, d) / math.sqrt(d), rnd(d, fs) / math.sqrt(fs)
    return {n: v.bfloat16() for n, v in t.items()}


def write(cfg, tens, path):
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file({n: v.contiguous() for n, v in tens.items()}, str(path / "model.safetensors"))
    return path


def rel(a, b):
    """Relative error of logits or activations (Frobenius)."""
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).norm() / (b.norm() + 1e-30)).item()


def worst_row(a, b):
    """Largest error of a row relative to the typical row norm: one wrong row among many shows."""
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).norm(dim=-1).max() / b.norm(dim=-1).mean()).item()


def worst_relative_row(a, b):
    """Largest error of a row relative to its own norm (rows of very different size, e.g. averages over 1 to n values)."""
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).norm(dim=-1) / (b.norm(dim=-1) + 1e-30)).max().item()


def row_errors(a, b):
    """Error of every row relative to the typical row norm."""
    a, b = a.double().cpu(), b.double().cpu()
    return (a - b).norm(dim=-1) / b.norm(dim=-1).mean()
