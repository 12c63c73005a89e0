"""Serving throughput of the Zafopel family beside the Dulisun family at equal size, whole steps and kernel by kernel.

    python bench.py --serve zafopel               (or: python -m rpeg_b200.engine.serve_bench_latent --sizes 2b,7b --layers 4)

Equal width, heads, value width, experts, chosen experts, parameters per expert and vocabulary. Zafopel layers alternate between causal ones
(queries through a latent, sink) and sliding ones, the last of four reads an earlier layer's latents; every layer has a mixture. Reports what
``serve_bench`` reports; each kernel of a Zafopel layer stands beside the like kernel of the Dulisun layer.
"""
from __future__ import annotations

import argparse
import json
import sys
from typing import List, Optional

import torch

from . import serve_bench as S

SIZES = {
    "2b": dict(width=2048, heads=16, dim=128, rot=64, rank=512, q_rank=768, window=8192, experts=32, top=4, ff=1024, vocab=32000, kv=4, groups=4, keep=2),
    "7b": dict(width=4096, heads=32, dim=128, rot=64, rank=512, q_rank=1536, window=8192, experts=64, top=6, ff=1024, vocab=32000, kv=8, groups=8, keep=3),
}


def build(size: str, layers: int, dev):
    from ..models.dulisun import AttentionMixer, DecoderLayer, DulisunConfig, DulisunModel, ExpertMixture
    from ..models.llama import LlamaConfig, LlamaModel
    from ..models.zafopel import InputScaledMixture, LatentMixer, ParallelLayer, ZafopelConfig, ZafopelModel
    s = SIZES[size]
    scale = (s["dim"] + s["rot"]) ** -0.5
    mixture = InputScaledMixture(s["experts"], s["top"], s["ff"])
    made = []
    for i in range(layers):
        common = dict(heads=s["heads"], dim=s["dim"], rot_dim=s["rot"], vdim=s["dim"], kv_rank=s["rank"], scale=scale)
        m = LatentMixer(**common, window=s["window"], kv_from=i - 2 if i % 4 == 3 else None) if i % 2 else LatentMixer(**common, q_rank=s["q_rank"], sink=True)
        made.append(ParallelLayer(m, mixture))
    z = ZafopelModel(ZafopelConfig(s["width"], s["vocab"], tuple(made), max_pos=16384), dev, seed=1)
    # a gated expert has three matrices, one without gate two
    mix = ExpertMixture(s["experts"], s["top"], s["ff"] * 3 // 2, 0, s["groups"], s["keep"])
    d = DulisunModel(DulisunConfig(s["width"], s["vocab"], (DecoderLayer(AttentionMixer(s["heads"], s["kv"], s["dim"], s["dim"] ** -0.5, s["window"], s["rot"],
                                                                                          10000.0), mix),) * layers, max_pos=16384), dev, seed=1)
    ll = LlamaModel(LlamaConfig(n_layers=layers, d_model=s["width"], d_ff=s["ff"] * s["top"], n_heads=s["heads"], n_kv_heads=s["kv"], head_dim=s["dim"],
                                vocab=s["vocab"], max_pos=16384, tie_embeddings=True), dev, seed=1)
    return z, d, ll


def prefill_kernels(tab: S.Table, z, d, ll, T: int) -> None:
    from ..ops import kernels as K
    S.prefill_kernels(tab, d, ll, T)                         # the like kernels
    dev, w = z.device, z.cfg.width
    m, e = z.cfg.layers[0].mixer, z.cfg.layers[0].mlp
    ph = f"prefill T={T}"
    i32, bf = dict(dtype=torch.int32, device=dev), dict(dtype=torch.bfloat16, device=dev)
    pos, slot, cu, lo = torch.arange(T, **i32), torch.zeros(T, **i32), torch.tensor([0, T], **i32), torch.zeros(1, **i32)
    pages = -(-T // K.KV_PAGE)
    table = torch.arange(1, 1 + pages, **i32).view(1, -1)
    R = range(2)
    layers = [0, 2 if z.cfg.n_layers > 2 else 0]             # causal layers of equal shape
    p = [{n[len(f"l{i}."):]: t for n, t in z.p.items() if n.startswith(f"l{i}.")} for i in layers]
    W, H, N = m.row_width, m.heads, m.heads * (m.dim_p + m.vdim_p)
    cos_t, sin_t = z._tables[(m.rot_base, m.rot_dim)]
    xb = [torch.randn(T, w, **bf) for _ in R]
    x32 = [torch.randn(T, w, device=dev) for _ in R]
    cache = [torch.randn(pages + 1, 1, K.KV_PAGE, W, **bf) for _ in R]
    n_in = m.q_in + m.kv_in

    def gemm(name, a, b, like):
        M, Kd, n = a[0].shape[0], a[0].shape[1], b[0].shape[0]
        tab.add(ph, name, [lambda i=i: K.gemm(a[i], b[i]) for i in R], 2 * (M * Kd + n * Kd + M * n), 2.0 * M * Kd * n, like=like)

    gemm("z input projection gemm", xb, [q["w_in"][:n_in] for q in p], "qk gemm")
    proj = [torch.randn(T, n_in, **bf) for _ in R]
    cq = [torch.randn(T, m.q_rank_p, **bf) for _ in R]
    tab.add(ph, "z latent norms + rotation + append", [lambda i=i: K.latent_rows(proj[i], pos, slot, cos_t, sin_t, m.rot_dim, m.rot_p, 1e-6,
            q_latent=(0, m.q_rank, p[i]["q_norm"], cq[i]), kv=(m.q_in, m.kv_rank, p[i]["kv_norm"], cache[i], table)) for i in R], 4 * T * n_in, like="rotary + unit norm + append")
    gemm("z query gemm", cq, [q["w_uq"] for q in p], "qk gemm")
    qs = [torch.randn(T, H, m.head_width, **bf) for _ in R]
    tab.add(ph, "z query rotation", [lambda i=i: K.latent_rows(qs[i].view(T, -1), pos, slot, cos_t, sin_t, m.rot_dim, m.rot_p, 1e-6,
            queries=(0, H, m.dim_p, None, qs[i][:, :, m.dim_p:])) for i in R], 4 * T * H * m.rot_p, like="rotary + unit norm + append")
    tab.add(ph, "z gather rows", [lambda i=i: K.latent_gather(cache[i], table, slot, cu, cu, lo, T) for i in R], 4 * T * W, like="dispatch")
    rows = [torch.randn(T, W, **bf) for _ in R]
    gemm("z key/value gemm", [r[:, : m.rank_p] for r in rows], [q["w_ukv"] for q in p], "qk gemm")
    kv = [torch.randn(T, N, **bf) for _ in R]
    short = max(128, T // 4)
    for window in (0, short):
        pairs = sum(min(t + 1, window or T) for t in range(T))
        tab.add(ph, "z prompt attention" + (f", window {window}" if window else ""), [lambda i=i: K.latent_prefill(qs[i], kv[i], rows[i], m.dim_p, m.vdim_p, m.rank_p, cu, pos, cu,
                lo, T, window=window, scale=m.scale, sink=z.sink[0]) for i in R], 2 * T * (H * m.head_width + N + m.rot_p + H * m.vdim_p), 2.0 * pairs * H * (m.dim + m.rot_dim + m.vdim),
                like=f"paged prefill attention, chunk {short if window else T}")
    att = [torch.randn(T, H * m.vdim_p, **bf) for _ in R]
    gemm("z o gemm", att, [q["wo"] for q in p], "qk gemm")
    del att, kv, rows, qs, proj
    router = [q["w_in"][n_in:] for q in p]
    lg = [K.gemm(xb[i], router[i], out_dtype=torch.float32) for i in R]
    tab.add(ph, "z router gemm", [lambda i=i: K.gemm(xb[i], router[i], out_dtype=torch.float32) for i in R], 2 * T * w + 4 * T * e.experts, 2.0 * T * w * e.experts, like="router gemm")
    counts = torch.zeros(e.experts, **i32)
    tab.add(ph, "z route", [lambda i=i: K.moe_route(lg[i], e.experts, e.top, counts, sigmoid=True) for i in R], 4 * T * (e.experts + 3 * e.top), like="route")
    rt = []
    for i in R:
        c = torch.zeros(e.experts, **i32)
        ids, wts, tk = K.moe_route(lg[i], e.experts, e.top, c, sigmoid=True)
        rt.append((ids, wts, tk, c, K.moe_dispatch(xb[i], ids, wts, tk, c, e.experts, weigh_inputs=True)))
    tab.add(ph, "z dispatch with weights", [lambda i=i: K.moe_dispatch(xb[i], *rt[i][:4], e.experts, weigh_inputs=True) for i in R], 2 * T * w * (1 + e.top), like="dispatch")
    n = T * e.top
    gate_up = lambda i: K.moe_gemm(rt[i][4].x_sorted, p[i]["w_gate_up"], rt[i][4], e.experts, 0, act="swiglu")  # noqa: E731
    tab.add(ph, "z experts gate/up gemm + swiglu", [lambda i=i: gate_up(i) for i in R], 2 * (n * w + e.experts * 2 * e.ff * w + n * e.ff), 4.0 * n * w * e.ff, like="experts up gemm + gelu")
    act = [gate_up(i) for i in R]
    down = lambda i: K.moe_gemm(act[i], p[i]["w_down"], rt[i][4], e.experts, 0)  # noqa: E731
    tab.add(ph, "z experts down gemm", [lambda i=i: down(i) for i in R], 2 * (n * e.ff + e.experts * e.ff * w + n * w), 2.0 * n * w * e.ff, like="experts down gemm")
    ys = [K.MoEOutput(down(i), rt[i][4].row_of, None, 0) for i in R]
    tab.add(ph, "z stream update + expert sum + norm", [lambda i=i: K.stream_update(xb[i], ys[i], z.alpha[0], p[i]["norm1"], p[i]["norm1.b"], x32[i]) for i in R],
            T * w * (2 * e.top + 12), like="expert sum + norm + fp32 residual")
    del ys, act, rt
    ff = e.ff * e.top                                       # a dense feed-forward of the chosen experts' size
    wu = [torch.randn(ff, w, **bf) for _ in R]
    tab.add(ph, "z dense up gemm + relu2", [lambda i=i: K.ff_first(xb[i], wu[i], "relu2") for i in R], 2 * (T * w + ff * w + T * ff), 2.0 * T * w * ff, like="experts up gemm + gelu")


def decode_kernels(tab: S.Table, z, d, ll, B: int, ctx: int) -> None:
    from ..ops import kernels as K
    S.decode_kernels(tab, d, ll, B, ctx)
    dev, w = z.device, z.cfg.width
    m, e = z.cfg.layers[0].mixer, z.cfg.layers[0].mlp
    ph = f"decode B={B} ctx={ctx}"
    i32, bf = dict(dtype=torch.int32, device=dev), dict(dtype=torch.bfloat16, device=dev)
    pages = -(-(ctx + 1) // K.KV_PAGE)
    table = torch.arange(1, 1 + B * pages, **i32).view(B, pages)
    pos, slot, lens = torch.full((B,), ctx, **i32), torch.arange(B, **i32), torch.full((B,), ctx + 1, **i32)
    layers = [i for i, l in enumerate(z.cfg.layers) if l.mixer.q_rank]
    p = [{n[len(f"l{i}."):]: t for n, t in z.p.items() if n.startswith(f"l{i}.")} for i in layers]
    R = range(len(layers))
    L = [i for _ in range(8) for i in R]
    W, H = m.row_width, m.heads
    cos_t, sin_t = z._tables[(m.rot_base, m.rot_dim)]
    cache = [torch.randn(B * pages + 1, 1, K.KV_PAGE, W, **bf) for _ in range(4)]
    C = [i for _ in range(4) for i in range(4)]
    ws, ws1 = z._workspace(), z._workspace(1)
    h, x32 = torch.randn(B, w, **bf), torch.randn(B, w, device=dev)
    K.set_pdl(True)

    def gemm(name, a, key, like, space=ws):
        ws_ = [q[key] for q in p]
        tab.add(ph, name, [lambda i=i: K.gemm_partials(a, ws_[i], space) for i in L], 2.0 * ws_[0].numel(), like=like)
        return K.gemm_partials(a, ws_[0], space)

    proj = gemm("z input projection gemm (split-K)", h, "w_in", "qk gemm (split-K)")
    cq = torch.randn(B, m.q_rank_p, **bf)
    tab.add(ph, "z latent norms + rotation + append", [lambda i=i: K.latent_rows(proj, pos, slot, cos_t, sin_t, m.rot_dim, m.rot_p, 1e-6,
            q_latent=(0, m.q_rank, p[0]["q_norm"], cq), kv=(m.q_in, m.kv_rank, p[0]["kv_norm"], cache[i], table)) for i in C], (4.0 * proj.splits + 2) * B * (m.q_in + m.kv_in),
            like="rotary + unit norm + append")
    qp = gemm("z query gemm (split-K)", cq, "w_uq", "qk gemm (split-K)", ws1)
    nope, wide = torch.randn(B, H * m.dim_p, **bf), torch.randn(B, H, W, **bf)
    tab.add(ph, "z query rotation", [lambda: K.latent_rows(qp, pos, slot, cos_t, sin_t, m.rot_dim, m.rot_p, 1e-6, queries=(0, H, m.dim_p, nope, wide[:, :, m.rank_p:])) for _ in C],
            (4.0 * qp.splits + 2) * B * m.q_width, like="rotary + unit norm + append")
    maps = [z._kv_maps(i) for i in layers]
    avg, out = torch.randn(B, H, m.rank_p, **bf), torch.empty(B, H, m.vdim_p, **bf)
    tab.add(ph, "z queries through key maps", [lambda i=i: K.head_gemm(nope.view(B, H, -1), maps[i][0], wide[:, :, : m.rank_p], transposed=True) for i in L],
            2.0 * (H * m.dim_p * m.rank_p + B * H * (m.dim_p + m.rank_p)), like="llama o gemm (split-K)")
    scratch = z._split_buffer(B, pages)
    ns = z._nsplit(m, B, pages)
    tab.add(ph, "z latent attention" + (f" + merge of {ns}" if ns > 1 else ""), [lambda i=i: K.latent_decode(wide, cache[i], m.rank_p, table, slot, pos, scale=m.scale, lens=lens, sink=z.sink[0],
            nsplit=ns, scratch=scratch) for i in C], 2.0 * B * (ctx + 1) * W, 2.0 * B * (ctx + 1) * H * (W + m.rank_p), like="rows attention")
    tab.add(ph, "z averages through value maps", [lambda i=i: K.head_gemm(avg, maps[i][1], out) for i in L],
            2.0 * (H * m.vdim_p * m.rank_p + B * H * (m.vdim_p + m.rank_p)), like="llama o gemm (split-K)")
    po = gemm("z o gemm (split-K)", out.view(B, -1), "wo", "llama o gemm (split-K)")
    rt = []
    for i in R:
        c = torch.zeros(e.experts, **i32)
        ids, wts, tk = K.moe_route(torch.randn(B, e.experts, device=dev), e.experts, e.top, c, sigmoid=True)
        rt.append((ids, wts, tk, c, K.moe_dispatch(h, ids, wts, tk, c, e.experts, weigh_inputs=True)))
    c0, lg = torch.zeros(e.experts, **i32), torch.randn(B, e.experts, device=dev)
    tab.add(ph, "z route", [lambda: K.moe_route(lg, e.experts, e.top, c0, sigmoid=True) for _ in L], 4.0 * B * (e.experts + 3 * e.top), like="route")
    tab.add(ph, "z dispatch with weights", [lambda i=i: K.moe_dispatch(h, *rt[i][:4], e.experts, weigh_inputs=True) for i in L], 2.0 * B * w * (1 + e.top), like="dispatch")
    used = sum(int((r[3] > 0).sum()) for r in rt) / len(rt)
    gate_up = lambda i: K.moe_gemm(rt[i][4].x_sorted, p[i]["w_gate_up"], rt[i][4], e.experts, 0, act="swiglu")  # noqa: E731
    tab.add(ph, "z experts gate/up gemm + swiglu", [lambda i=i: gate_up(i) for i in L], used * 4.0 * e.ff * w, like="experts up gemm + gelu")
    act = [gate_up(i) for i in R]
    tab.add(ph, "z experts down gemm", [lambda i=i: K.moe_gemm(act[i], p[i]["w_down"], rt[i][4], e.experts, 0) for i in L], used * 2.0 * e.ff * w, like="experts down gemm")
    ys = K.MoEOutput(K.moe_gemm(act[0], p[0]["w_down"], rt[0][4], e.experts, 0), rt[0][4].row_of, None, 0)
    tab.add(ph, "z stream update + expert sum + norm", [lambda: K.stream_update(po, ys, z.alpha[0], p[0]["norm1"], p[0]["norm1.b"], x32) for _ in L],
            B * w * (4.0 * po.splits + 2.0 * e.top + 10), like="expert sum + norm + fp32 residual")
    # a layer with a dense feed-forward of the chosen experts' size: its first product rides on the input projection
    ff = e.ff * e.top
    wu = [torch.randn(m.q_in + m.kv_in + ff, w, **bf) for _ in range(4)]
    tab.add(ph, "z input projection + dense up gemm (split-K)", [lambda i=i: K.gemm_partials(h, wu[i], ws) for i in C], 2.0 * wu[0].numel(), like="llama gate/up gemm (split-K)")
    pd, fa = K.gemm_partials(h, wu[0], ws), torch.empty(B, ff, **bf)
    tab.add(ph, "z latent norms + rotation + append + relu2", [lambda i=i: K.latent_rows(pd, pos, slot, cos_t, sin_t, m.rot_dim, m.rot_p, 1e-6,
            q_latent=(0, m.q_rank, p[0]["q_norm"], cq), kv=(m.q_in, m.kv_rank, p[0]["kv_norm"], cache[i], table), ff=(m.q_in + m.kv_in, fa)) for i in C],
            (4.0 * pd.splits + 2) * B * (m.q_in + m.kv_in + ff), like="rotary + unit norm + append")


def run(sizes: List[str], layers: int, kernels: bool = True) -> dict:
    from ..ops import kernels as K
    dev = torch.device("cuda:0")
    torch.cuda.set_device(0)
    pk = S.peaks()
    out = {"impl": "ours", "metric": "serve_tokens_per_sec", "unit": "tokens/s", "higher_is_better": True, "data": "synthetic", "dtype": "bf16", "n_gpus": 1,
           "peaks": pk, "layers": layers, "sizes": {}}
    for size in sizes:
        with torch.no_grad():
            z, d, ll = build(size, layers, dev)
            res = {"shape": SIZES[size], "params": [z.cfg.n_params(), d.cfg.n_params()], "prefill": [], "decode": [], "kernels": []}
            for rows, length in S.PREFILL:
                a, b = S.prefill_rate(z, rows, length), S.prefill_rate(d, rows, length)
                res["prefill"].append({"rows": rows, "length": length, "zafopel": round(a), "dulisun": round(b), "ratio": round(a / b, 3)})
            for batch, ctx in S.DECODE:
                a, b = S.decode_rate(z, batch, ctx), S.decode_rate(d, batch, ctx)
                res["decode"].append({"batch": batch, "ctx": ctx, "zafopel": round(a), "dulisun": round(b), "ratio": round(a / b, 3)})
            if kernels:
                tab = S.Table(pk)
                prefill_kernels(tab, z, d, ll, 8192)
                decode_kernels(tab, z, d, ll, 64, 2048)
                decode_kernels(tab, z, d, ll, 8, 2048)
                res["kernels"] = tab.rows
            K.check_status()
            out["sizes"][size] = res
            del z, d, ll
            torch.cuda.empty_cache()
    first = out["sizes"][sizes[-1]]
    out["value"] = next(r["zafopel"] for r in first["decode"] if r["batch"] == 64)
    return out


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(description="Serving throughput of the Zafopel family beside the Dulisun family")
    ap.add_argument("--sizes", default="2b,7b")
    ap.add_argument("--layers", type=int, default=4)
    ap.add_argument("--no-kernels", action="store_true")
    args = ap.parse_args(argv)
    print(json.dumps(run(args.sizes.split(","), args.layers, not args.no_kernels)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
