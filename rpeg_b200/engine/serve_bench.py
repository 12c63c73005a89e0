"""Serving throughput of the Dulisun family beside the Llama family at equal size, whole steps and kernel by kernel.

    python bench.py --serve                       (or: python -m rpeg_b200.engine.serve_bench --sizes 2b,7b --layers 4)

``bench.py --serve zafopel`` (``engine/serve_bench_latent.py``) does the same for the Zafopel family beside this one.

Both models get the same width, heads, KV heads, head size and vocabulary; the Llama feed-forward is as wide as makes its
parameters equal to those a Dulisun token uses (chosen experts plus the shared one). Random weights, ``--layers`` layers of
the real size (a layer's rate does not depend on how many there are). Reported per size:

  prefill   tokens/s of the generator's prefill (K/V append included) for several batches of prompts
  decode    tokens/s of the generator's captured step (LM head and sampling included) for several batches and contexts
  kernels   time per launch, the roofline floor max(bytes / copy rate, FLOPs / matrix rate) and the fraction reached, each
            kernel of the Dulisun layer beside the like kernel of the Llama layer, and the quotient of the two fractions

Kernel times are CUDA-graph replays of launches that rotate over the layers' own weights and caches (beyond L2 where the
workload itself is beyond it). Prints one JSON object.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Callable, Dict, List, Optional

import torch

SIZES = {
    "2b": dict(width=2048, heads=16, kv=4, dim=128, window=8192, rot=64, experts=32, top=4, groups=4, keep=2, ff=1024, shared=1024, vocab=32000),
    "7b": dict(width=4096, heads=32, kv=8, dim=128, window=8192, rot=64, experts=64, top=6, groups=8, keep=3, ff=1408, shared=2816, vocab=32000),
}
PREFILL = ((8, 1024), (1, 8192))
DECODE = ((1, 2048), (8, 2048), (64, 2048), (256, 1024))


def peaks() -> Dict[str, float]:
    f = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if f.exists():
        p = json.loads(f.read_text())
        return {"hbm_gbs": float(p["hbm_gbs"]), "tflops": float(p["bf16_tflops"]), "source": "measured"}
    return {"hbm_gbs": 6650.0, "tflops": 1590.0, "source": "fallback"}


def build(size: str, layers: int, dev):
    from ..models.dulisun import AttentionMixer, DecoderLayer, DulisunConfig, DulisunModel, ExpertMixture
    from ..models.llama import LlamaConfig, LlamaModel
    s = SIZES[size]
    mixer = AttentionMixer(s["heads"], s["kv"], s["dim"], s["dim"] ** -0.5, s["window"], s["rot"], 10000.0)
    mix = ExpertMixture(s["experts"], s["top"], s["ff"], s["shared"], s["groups"], s["keep"])
    d = DulisunModel(DulisunConfig(s["width"], s["vocab"], (DecoderLayer(mixer, mix),) * layers, max_pos=16384), dev, seed=1)
    ff = -(-(2 * (s["top"] * s["ff"] + s["shared"])) // (3 * 128)) * 128
    ll = LlamaModel(LlamaConfig(n_layers=layers, d_model=s["width"], d_ff=ff, n_heads=s["heads"], n_kv_heads=s["kv"], head_dim=s["dim"],
                                vocab=s["vocab"], max_pos=16384, tie_embeddings=True), dev, seed=1)
    return d, ll


def time_us(fns: List[Callable[[], object]], rounds: int = 5) -> float:
    """Microseconds per launch: the list captured once as a graph, ``rounds`` replays timed with events, the median taken."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for f in fns:
            f()
    torch.cuda.current_stream().wait_stream(side)
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for f in fns:
            f()
    for _ in range(3):
        g.replay()
    out = []
    for _ in range(rounds):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        g.replay()
        b.record()
        b.synchronize()
        out.append(a.elapsed_time(b) * 1e3 / len(fns))
    del g
    return sorted(out)[len(out) // 2]


# ---------------------------------------------------------------------------------------------------- whole steps
def prefill_rate(model, rows: int, length: int) -> float:
    from .generation import PAGE, Generator
    gen = Generator(model, max_slots=max(rows, 1), max_seq_len=length + PAGE, kv_budget_bytes=40e9, use_graphs=False)
    n = gen.pages_per_row
    gen.page_table.copy_(torch.arange(1, 1 + gen.max_slots * n, dtype=torch.int32, device=gen.dev).view(gen.max_slots, n))
    prompts = [torch.randint(3, model.cfg.vocab, (length,), dtype=torch.int32, device=gen.dev) for _ in range(rows)]
    ms = []
    for i in range(6):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        gen._prefill(prompts, list(range(rows)))
        b.record()
        b.synchronize()
        if i >= 3:
            ms.append(a.elapsed_time(b))
    return rows * length / (sorted(ms)[1] / 1e3)


def decode_rate(model, batch: int, ctx: int, iters: int = 30) -> float:
    from .generation import Generator
    gen = Generator(model, max_slots=batch, max_seq_len=ctx + 128, kv_budget_bytes=60e9)
    n = gen.pages_per_row
    gen.page_table.copy_(torch.arange(1, 1 + gen.max_slots * n, dtype=torch.int32, device=gen.dev).view(gen.max_slots, n))
    gen.kv_storage.normal_()
    gen.out_tok = torch.zeros((gen.max_slots, 4096), dtype=torch.int32, device=gen.dev)
    gen.out_lp = torch.zeros((gen.max_slots, 4096), dtype=torch.float32, device=gen.dev)

    def reset():
        gen.active.fill_(1)
        gen.gen_count.fill_(1)
        gen.seq_len.fill_(ctx + 1)
        gen.pos.fill_(ctx)
        gen.token.random_(3, model.cfg.vocab)

    gen.eos_id = -1
    reset()
    for _ in range(4):
        gen._step(batch, 1.0, False, 0)
    reset()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        gen._step(batch, 1.0, False, 0)
    b.record()
    b.synchronize()
    return batch * iters / (a.elapsed_time(b) / 1e3)


# ---------------------------------------------------------------------------------------------------- kernels
class Table:
    def __init__(self, pk: Dict[str, float]):
        self.pk, self.rows = pk, []

    def add(self, phase: str, name: str, fns, nbytes: float, flops: float = 0.0, like: Optional[str] = None, rounds: int = 5) -> float:
        us = time_us(fns, rounds)
        floor = max(nbytes / (self.pk["hbm_gbs"] * 1e3), flops / (self.pk["tflops"] * 1e6))
        row = {"phase": phase, "kernel": name, "us": round(us, 2), "floor_us": round(floor, 3), "fraction": round(floor / us, 4)}
        if like is not None:
            ref = next(r for r in self.rows if r["phase"] == phase and r["kernel"] == like)
            row["like"] = like
            row["times_further_from_roofline"] = round(ref["floor_us"] / ref["us"] * us / floor, 2)
        self.rows.append(row)
        return us


def prefill_kernels(tab: Table, d, ll, T: int) -> None:
    from ..ops import kernels as K
    dev, n = d.device, d.cfg.n_layers
    m, e, w = d.cfg.layers[0].mixer, d.cfg.layers[0].mlp, d.cfg.width
    lc = ll.cfg
    H, G, hd = m.heads, m.kv_heads, m.dim
    ph = f"prefill T={T}"
    i32 = dict(dtype=torch.int32, device=dev)
    bf = dict(dtype=torch.bfloat16, device=dev)
    pos, slot, cu = torch.arange(T, **i32), torch.zeros(T, **i32), torch.tensor([0, T], **i32)
    pages = -(-T // K.KV_PAGE)
    table = torch.arange(1, 1 + pages, **i32).view(1, -1)
    R = range(max(2, min(n, 4)))
    kc = [torch.randn(pages + 1, G, K.KV_PAGE, hd, **bf) for _ in R]
    vc = [torch.randn(pages + 1, G, K.KV_PAGE, hd, **bf) for _ in R]
    xb = [torch.randn(T, w, **bf) for _ in R]
    res = [torch.randn(T, w, **bf) for _ in R]
    x32 = [torch.randn(T, w, device=dev) for _ in R]
    qkv = [torch.randn(T, lc.qkv_width, **bf) for _ in R]
    qk = [torch.randn(T, (H + G) * hd, **bf) for _ in R]
    q = [torch.empty(T, H * hd, **bf) for _ in R]
    cos_t, sin_t = d._tables[(m.rot_base, m.rot_dims)]

    tab.add(ph, "llama rmsnorm + residual", [lambda i=i: K.rmsnorm_fwd(xb[i], ll.p["l0.attn_norm"], 1e-5, residual=res[i], want_sum=True) for i in R], T * w * 8)
    tab.add(ph, "norm + fp32 residual", [lambda i=i: K.residual_norm(xb[i], d.p["l0.norm1"], 1e-6, w, x=x32[i]) for i in R], T * w * 12, like="llama rmsnorm + residual")
    tab.add(ph, "llama qkv gemm", [lambda i=i: K.gemm(xb[i], ll.p[f"l{i % n}.wqkv"]) for i in R], 2 * (T * w + lc.qkv_width * w + T * lc.qkv_width), 2.0 * T * w * lc.qkv_width)
    tab.add(ph, "qk gemm", [lambda i=i: K.gemm(xb[i], d.p[f"l{i % n}.wqk"]) for i in R], 2 * (T * w + (H + G) * hd * w + T * (H + G) * hd), 2.0 * T * w * (H + G) * hd, like="llama qkv gemm")

    def llama_rope(i):
        K.rope_(qkv[i], pos, ll.cos_t, ll.sin_t, 0, H, hd)
        K.rope_(qkv[i], pos, ll.cos_t, ll.sin_t, lc.q_width, G, hd)
        K.kv_append(qkv[i], lc.q_width, lc.q_width + lc.kv_width, slot, pos, table, kc[i], vc[i], G, hd)
    tab.add(ph, "llama rope + append (3 launches)", [lambda i=i: llama_rope(i) for i in R], 4 * T * (H + G) * hd + 4 * T * 2 * G * hd)
    tab.add(ph, "rotary + unit norm + append", [lambda i=i: K.rotary_append(qk[i], q[i], 0, H * hd, H * hd, slot, pos, cos_t, sin_t, table, kc[i], vc[i], H, hd,
                                                                          m.rot_dims, 1e-6) for i in R], 2 * T * ((H + G) * hd + H * hd + 2 * G * hd), like="llama rope + append (3 launches)")
    pairs = T * (T + 1) / 2
    tab.add(ph, "llama flash attention", [lambda i=i: K.flash_attn_fwd(qkv[i], 0, lc.q_width, lc.q_width + lc.kv_width, cu, T, H, G, hd) for i in R],
            2 * T * (lc.qkv_width + H * hd), 4.0 * pairs * H * hd)
    short = max(128, T // 4)
    cu4 = torch.arange(0, T + 1, short, **i32)
    tab.add(ph, f"llama flash attention, sequences of {short}", [lambda i=i: K.flash_attn_fwd(qkv[i], 0, lc.q_width, lc.q_width + lc.kv_width, cu4, short, H, G, hd) for i in R],
            2 * T * (lc.qkv_width + H * hd), 4.0 * (T // short) * short * (short + 1) / 2 * H * hd)
    for window in (T, short):
        vis = sum(min(T - c, window) * (min(T - c, window) + 1) / 2 for c in range(0, T, window))
        tab.add(ph, f"paged prefill attention, chunk {window}", [lambda i=i: K.window_prefill(q[i], kc[i], vc[i], table, cu, pos, slot, T, H, window=window,
                scale=hd ** -0.5, sink=d.sink[0]) for i in R], 2 * T * (2 * H + 2 * G) * hd, 4.0 * vis * H * hd,
                like="llama flash attention" if window == T else f"llama flash attention, sequences of {short}")
    f = lc.d_ff
    tab.add(ph, "llama gate/up gemm + swiglu", [lambda i=i: K.gemm_swiglu(xb[i], ll.p[f"l{i % n}.w_gate_up"]) for i in R], 2 * (T * w + 2 * f * w + T * f), 4.0 * T * w * f)
    act = [torch.randn(T, f, **bf) for _ in R]
    tab.add(ph, "llama down gemm", [lambda i=i: K.gemm(act[i], ll.p[f"l{i % n}.w_down"]) for i in R], 2 * (T * w + f * w + T * f), 2.0 * T * w * f)
    del act
    counts = torch.zeros(e.experts, **i32)
    lg = [K.gemm(xb[i], d.p[f"l{i % n}.router"], out_dtype=torch.float32) for i in R]
    tab.add(ph, "router gemm", [lambda i=i: K.gemm(xb[i], d.p[f"l{i % n}.router"], out_dtype=torch.float32) for i in R], 2 * T * w + 4 * T * e.experts, 2.0 * T * w * e.experts,
            like="llama down gemm")
    tab.add(ph, "route", [lambda i=i: K.moe_route(lg[i], e.experts, e.top, counts, n_groups=e.groups, keep_groups=e.keep) for i in R], 4 * T * (e.experts + 3 * e.top),
            like="llama rmsnorm + residual")
    rt = []
    for i in R:
        c = torch.zeros(e.experts, **i32)
        ids, wts, tk = K.moe_route(lg[i], e.experts, e.top, c, n_groups=e.groups, keep_groups=e.keep)
        rt.append((ids, wts, tk, c, K.moe_dispatch(xb[i], ids, wts, tk, c, e.experts)))
    tab.add(ph, "dispatch", [lambda i=i: K.moe_dispatch(xb[i], *rt[i][:4], e.experts) for i in R], 2 * T * w * (1 + e.top), like="llama rmsnorm + residual")
    rows, seg = T * (e.top + e.n_shared), e.segments
    tab.add(ph, "experts up gemm + gelu", [lambda i=i: K.moe_gemm(rt[i][4].x_sorted, d.p[f"l{i % n}.w_up"], rt[i][4], e.experts, e.n_shared, shared_x=xb[i], act="gelu") for i in R],
            2 * (T * w * (1 + e.top) + seg * e.ff * w + rows * e.ff), 2.0 * rows * w * e.ff, like="llama gate/up gemm + swiglu")
    up = [K.moe_gemm(rt[i][4].x_sorted, d.p[f"l{i % n}.w_up"], rt[i][4], e.experts, e.n_shared, shared_x=xb[i], act="gelu") for i in R]
    tab.add(ph, "experts down gemm", [lambda i=i: K.moe_gemm(up[i], d.p[f"l{i % n}.w_down"], rt[i][4], e.experts, e.n_shared) for i in R],
            2 * (rows * e.ff + seg * e.ff * w + rows * w), 2.0 * rows * w * e.ff, like="llama down gemm")
    ys = [K.MoEOutput(K.moe_gemm(up[i], d.p[f"l{i % n}.w_down"], rt[i][4], e.experts, e.n_shared), rt[i][4].row_of, rt[i][4].weights, e.n_shared) for i in R]
    tab.add(ph, "expert sum + norm + fp32 residual", [lambda i=i: K.residual_norm(ys[i], d.p["l0.norm2"], 1e-6, w, x=x32[i]) for i in R], T * w * (2 * (e.top + e.n_shared) + 10),
            like="llama rmsnorm + residual")


def decode_kernels(tab: Table, d, ll, B: int, ctx: int) -> None:
    from ..ops import kernels as K
    dev, n = d.device, d.cfg.n_layers
    m, e, w = d.cfg.layers[0].mixer, d.cfg.layers[0].mlp, d.cfg.width
    lc = ll.cfg
    H, G, hd, f = m.heads, m.kv_heads, m.dim, lc.d_ff
    ph = f"decode B={B} ctx={ctx}"
    i32 = dict(dtype=torch.int32, device=dev)
    bf = dict(dtype=torch.bfloat16, device=dev)
    pages = -(-(ctx + 1) // K.KV_PAGE)
    table = torch.arange(1, 1 + B * pages, **i32).view(B, pages)
    pos, slot, lens = torch.full((B,), ctx, **i32), torch.arange(B, **i32), torch.full((B,), ctx + 1, **i32)
    R = range(n)
    kc = [torch.randn(B * pages + 1, G, K.KV_PAGE, hd, **bf) for _ in R]
    vc = [torch.randn(B * pages + 1, G, K.KV_PAGE, hd, **bf) for _ in R]
    ws = d._workspace()
    h, x32, att = torch.randn(B, w, **bf), torch.randn(B, w, device=dev), torch.randn(B, H * hd, **bf)
    qkv, q = torch.randn(B, lc.qkv_width, **bf), torch.randn(B, H * hd, **bf)
    cos_t, sin_t = d._tables[(m.rot_base, m.rot_dims)]
    rep = 4
    nsp = 1 if B * H >= 296 else min(8, (296 + B * H - 1) // (B * H))
    K.set_pdl(True)
    L = [i for _ in range(rep) for i in R]

    def wbytes(rows, cols):
        return 2.0 * rows * cols

    tab.add(ph, "llama qkv gemm (split-K)", [lambda i=i: K.gemm_partials(h, ll.p[f"l{i}.wqkv"], ws) for i in L], wbytes(lc.qkv_width, w))
    tab.add(ph, "qk gemm (split-K)", [lambda i=i: K.gemm_partials(h, d.p[f"l{i}.wqk"], ws) for i in L], wbytes((H + G) * hd, w), like="llama qkv gemm (split-K)")
    parts = K.gemm_partials(h, ll.p["l0.wqkv"], ws)
    tab.add(ph, "llama rope + append", [lambda i=i: K.rope_kv_append_partials_(parts, qkv, 0, lc.q_width, lc.q_width + lc.kv_width, slot, pos, ll.cos_t, ll.sin_t, table, kc[i], vc[i], H, G, hd)
                                        for i in L], 4.0 * parts.splits * B * lc.qkv_width + 2.0 * B * lc.qkv_width)
    pq = K.gemm_partials(h, d.p["l0.wqk"], ws)
    tab.add(ph, "rotary + unit norm + append", [lambda i=i: K.rotary_append(pq, q, 0, H * hd, H * hd, slot, pos, cos_t, sin_t, table, kc[i], vc[i], H, hd, m.rot_dims, 1e-6) for i in L],
            4.0 * pq.splits * B * (H + G) * hd + 2.0 * B * (H + 2 * G) * hd, like="llama rope + append")
    kv_bytes = 2.0 * B * (ctx + 1) * G * hd * 2
    scr = torch.empty(max(1, K.decode_scratch_numel(B, H, nsp)), device=dev)
    tab.add(ph, "llama paged decode attention", [lambda i=i: K.paged_decode_attn(qkv, 0, kc[i], vc[i], table, lens, H, G, hd, hd ** -0.5, nsplit=nsp, scratch=scr) for i in L], kv_bytes)
    scratch, arrive = d._split_buffers(B, pages)
    tab.add(ph, "rows attention", [lambda i=i: K.rows_attn(q, kc[i], vc[i], table, slot, pos, H, window=m.window, scale=hd ** -0.5, lens=lens, sink=d.sink[0],
            nsplit=d._nsplit(m, B, pages), scratch=scratch, arrive=arrive) for i in L], kv_bytes, like="llama paged decode attention")
    tab.add(ph, "llama o gemm (split-K)", [lambda i=i: K.gemm_partials(att, ll.p[f"l{i}.wo"], ws) for i in L], wbytes(H * hd, w))
    po = K.gemm_partials(att, ll.p["l0.wo"], ws)
    tab.add(ph, "llama rmsnorm + residual", [lambda i=i: K.rmsnorm_fwd_partials(po, ll.p["l0.mlp_norm"], 1e-5, residual=h, want_sum=True) for i in L], B * w * (4.0 * po.splits + 6))
    tab.add(ph, "norm + fp32 residual", [lambda i=i: K.residual_norm(po, d.p["l0.norm1"], 1e-6, w, x=x32) for i in L], B * w * (4.0 * po.splits + 10), like="llama rmsnorm + residual")
    tab.add(ph, "llama gate/up gemm (split-K)", [lambda i=i: K.gemm_partials(h, ll.p[f"l{i}.w_gate_up"], ws) for i in L], wbytes(2 * f, w))
    pg = K.gemm_partials(h, ll.p["l0.w_gate_up"], ws)
    tab.add(ph, "llama swiglu", [lambda i=i: K.swiglu_fwd_partials(pg) for i in L], B * f * (8.0 * pg.splits + 2))
    act = torch.randn(B, f, **bf)
    tab.add(ph, "llama down gemm (split-K)", [lambda i=i: K.gemm_partials(act, ll.p[f"l{i}.w_down"], ws) for i in L], wbytes(f, w))
    tab.add(ph, "router gemm (split-K)", [lambda i=i: K.gemm_partials(h, d.p[f"l{i}.router"], ws) for i in L], wbytes(e.experts, w), like="llama o gemm (split-K)")
    # distinct routing per layer, as in a model; the experts that any row chose are the weights that must be read
    rt = []
    for i in R:
        c = torch.zeros(e.experts, **i32)
        lg = torch.randn(B, e.experts, device=dev)
        ids, wts, tk = K.moe_route(lg, e.experts, e.top, c, n_groups=e.groups, keep_groups=e.keep)
        rt.append((ids, wts, tk, c, K.moe_dispatch(h, ids, wts, tk, c, e.experts)))
    lg = torch.randn(B, e.experts, device=dev)
    c0 = torch.zeros(e.experts, **i32)
    tab.add(ph, "route", [lambda: K.moe_route(lg, e.experts, e.top, c0, n_groups=e.groups, keep_groups=e.keep) for _ in L], 4.0 * B * (e.experts + 3 * e.top), like="llama swiglu")
    tab.add(ph, "dispatch", [lambda i=i: K.moe_dispatch(h, *rt[i][:4], e.experts) for i in L], 2.0 * B * w * (1 + e.top), like="llama rmsnorm + residual")
    used = sum(int((r[3] > 0).sum()) for r in rt) / n + e.n_shared
    tab.add(ph, "experts up gemm + gelu", [lambda i=i: K.moe_gemm(rt[i][4].x_sorted, d.p[f"l{i}.w_up"], rt[i][4], e.experts, e.n_shared, shared_x=h, act="gelu") for i in L],
            used * wbytes(e.ff, w), like="llama gate/up gemm (split-K)")
    up = [K.moe_gemm(rt[i][4].x_sorted, d.p[f"l{i}.w_up"], rt[i][4], e.experts, e.n_shared, shared_x=h, act="gelu") for i in R]
    tab.add(ph, "experts down gemm", [lambda i=i: K.moe_gemm(up[i], d.p[f"l{i}.w_down"], rt[i][4], e.experts, e.n_shared) for i in L], used * wbytes(e.ff, w),
            like="llama down gemm (split-K)")
    ys = [K.MoEOutput(K.moe_gemm(up[i], d.p[f"l{i}.w_down"], rt[i][4], e.experts, e.n_shared), rt[i][4].row_of, rt[i][4].weights, e.n_shared) for i in R]
    tab.add(ph, "expert sum + norm + fp32 residual", [lambda i=i: K.residual_norm(ys[i], d.p["l0.norm2"], 1e-6, w, x=x32) for i in L], B * w * (2.0 * (e.top + e.n_shared) + 10),
            like="llama rmsnorm + residual")


def run(sizes: List[str], layers: int, kernels: bool = True) -> dict:
    from ..ops import kernels as K
    dev = torch.device("cuda:0")
    torch.cuda.set_device(0)
    pk = peaks()
    out = {"impl": "ours", "metric": "serve_tokens_per_sec", "unit": "tokens/s", "higher_is_better": True, "data": "synthetic", "dtype": "bf16", "n_gpus": 1,
           "peaks": pk, "layers": layers, "sizes": {}}
    for size in sizes:
        with torch.no_grad():
            d, ll = build(size, layers, dev)
            res = {"shape": SIZES[size], "llama_d_ff": ll.cfg.d_ff, "prefill": [], "decode": [], "kernels": []}
            for rows, length in PREFILL:
                a, b = prefill_rate(d, rows, length), prefill_rate(ll, rows, length)
                res["prefill"].append({"rows": rows, "length": length, "dulisun": round(a), "llama": round(b), "ratio": round(a / b, 3)})
            for batch, ctx in DECODE:
                a, b = decode_rate(d, batch, ctx), decode_rate(ll, batch, ctx)
                res["decode"].append({"batch": batch, "ctx": ctx, "dulisun": round(a), "llama": round(b), "ratio": round(a / b, 3)})
            if kernels:
                tab = Table(pk)
                prefill_kernels(tab, d, ll, 8192)
                decode_kernels(tab, d, ll, 64, 2048)
                decode_kernels(tab, d, ll, 8, 2048)
                res["kernels"] = tab.rows
            K.check_status()
            out["sizes"][size] = res
            del d, ll
            torch.cuda.empty_cache()
    first = out["sizes"][sizes[-1]]
    out["value"] = next(r["dulisun"] for r in first["decode"] if r["batch"] == 64)
    return out


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(description="Serving throughput of the Dulisun family beside the Llama family")
    ap.add_argument("--sizes", default="2b,7b")
    ap.add_argument("--layers", type=int, default=4)
    ap.add_argument("--no-kernels", action="store_true")
    args = ap.parse_args(argv)
    print(json.dumps(run(args.sizes.split(","), args.layers, not args.no_kernels)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
