"""GPU tests of the Dulisun family against the plain oracle: every mechanism alone, then the model through the generator's
cache, scheduler and entry points. fp32 runs are the sharp ones (a missing key, a wrong page or a lost sink is orders of
magnitude above their tolerance); bf16 kernels are also tested on inputs where single scores stand out."""
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

pytestmark = pytest.mark.gpu

import dulisun_cases as C  # noqa: E402
import dulisun_oracle as O  # noqa: E402
from rpeg_b200.engine import algorithms as A  # noqa: E402
from rpeg_b200.engine.generation import PAGE, Generator, page_elems  # noqa: E402
from rpeg_b200.engine.session import Session  # noqa: E402
from rpeg_b200.models.registry import load_model  # noqa: E402
from rpeg_b200.ops import checked  # noqa: E402
from rpeg_b200.ops import kernels as K  # noqa: E402

DT = (torch.float32, torch.bfloat16)
TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}
ATTN = {torch.float32: 2e-5, torch.bfloat16: 5e-3}        # scores, weights and sums are fp32: only the output is rounded
ROOT = Path(__file__).resolve().parent.parent


@pytest.fixture(autouse=True)
def _status():
    yield
    K.check_status()


def _pad(x, n):
    return torch.nn.functional.pad(x, (0, n - x.shape[-1])).contiguous()


# --------------------------------------------------------------------------- norms
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("rows,d", [(1, 5), (3, 100), (37, 256), (5, 1030), (2, 13000)])
def test_residual_norm_sources(cuda_device, dtype, rows, d):
    g = torch.Generator().manual_seed(d)
    dp = -(-d // 8) * 8
    dev, eps = cuda_device, 1e-3
    w, w2 = (_pad((0.5 * torch.randn(d, generator=g)).to(dtype), dp).to(dev) for _ in range(2))
    x0 = _pad(torch.randn(rows, d, generator=g), dp).to(dev)
    wd, w2d, xd = (t[..., :d].double().cpu() for t in (w, w2, x0))

    def check(got, want, tol=None):
        assert C.rel(got[:, :d], want) < (tol or TOL[dtype] / 3)
        assert got[:, d:].abs().sum() == 0

    src = _pad(torch.randn(rows, d, generator=g).to(dtype), dp).to(dev)
    want = O.norm(src[:, :d].double().cpu(), wd, eps)
    x = x0.clone()
    y = K.residual_norm(src, w, eps, d, x=x)
    check(x, xd + want, 1e-6)
    check(y, xd + want)
    # plain weights, no residual, no stream
    check(K.residual_norm(src, w, eps, d, add=False, zero_centered=False), O.rms(src[:, :d].double().cpu(), eps) * wd)
    # the next norm in the same launch, and the stream as the source
    x = x0.clone()
    check(K.residual_norm(src, w, eps, d, x=x, w2=w2), O.norm(xd + want, w2d, eps))
    check(K.residual_norm(x0, w, eps, d, add=False), O.norm(xd, wd, eps))
    # an embedding row starts the stream
    table = _pad(torch.randn(9, d, generator=g).to(dtype), dp).to(dev)
    ids = torch.randint(0, 9, (rows,), generator=g, dtype=torch.int32).to(dev)
    x = torch.full_like(x0, 7.0)
    K.residual_norm(table, w, eps, d, ids=ids, x=x, add=False)
    check(x, O.norm(table[ids.long(), :d].double().cpu(), wd, eps), 1e-6)
    # split-K partials
    buf = torch.zeros(3, rows, dp, device=dev)
    buf[..., :d] = torch.randn(3, rows, d, generator=g).to(dev)
    x = x0.clone()
    K.residual_norm(K.Partials(buf.view(-1), 3, rows, dp), w, eps, d, x=x)
    check(x, xd + O.norm(buf[..., :d].double().sum(0).cpu(), wd, eps), 1e-6)


# --------------------------------------------------------------------------- rotation and append
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,G,dim,rot,partials", [(6, 3, 20, 12, False), (3, 1, 96, 96, False), (4, 2, 200, 50, False), (5, 5, 256, 0, False),
                                                 (12, 2, 40, 2, True), (6, 2, 128, 64, True)])
def test_rotary_append(cuda_device, dtype, H, G, dim, rot, partials):
    if partials and dtype == torch.float32:
        pytest.skip("split-K partials belong to the bf16 path")
    g = torch.Generator().manual_seed(dim)
    dev, T, dp, eps, base = cuda_device, 70, -(-dim // 8) * 8, 1e-2, 300.0
    raw = torch.zeros(T, H + G, dp)
    raw[..., :dim] = torch.randn(T, H + G, dim, generator=g)
    raw = raw.to(dtype)
    slot = torch.tensor([0] * 40 + [1] * 30, dtype=torch.int32)
    pos = torch.cat([torch.arange(100, 140), torch.arange(3, 33)]).int()
    table = torch.tensor([[5, 2, 7], [1, 4, 0]], dtype=torch.int32)
    kc, vc = (torch.full((8, G, PAGE, dp), 9.0, dtype=dtype, device=dev) for _ in range(2))
    q_out = torch.zeros(T, H * dp, dtype=dtype, device=dev)
    cos_t, sin_t = K.rope_tables(256, rot, base, dev) if rot else (None, None)
    if partials:
        parts = torch.randn(2, T, (H + G) * dp, generator=g).view(2, T, H + G, dp)
        parts[..., dim:] = 0
        raw = parts.sum(0)
        src = K.Partials(parts.reshape(-1).to(dev), 2, T, (H + G) * dp)
    else:
        src = raw.view(T, -1).to(dev)
    K.rotary_append(src, q_out, 0, H * dp, H * dp, slot.to(dev), pos.to(dev), cos_t, sin_t, table.to(dev), kc, vc, H, dim, rot, eps)
    want = O.rms(O.rotate(raw[..., :dim].double(), pos, base, rot), eps)
    assert C.worst_row(q_out.view(T, H, dp)[..., :dim].reshape(T, -1), want[:, :H].reshape(T, -1)) < TOL[dtype]
    pages = table[slot.long(), pos.long() // PAGE].long()
    k_got, v_got = kc[pages, :, pos.long() % PAGE], vc[pages, :, pos.long() % PAGE]
    assert C.worst_row(k_got[..., :dim].reshape(T, -1), want[:, H:].reshape(T, -1)) < TOL[dtype]
    assert C.worst_row(v_got[..., :dim].reshape(T, -1), raw[:, H:, :dim].reshape(T, -1)) < TOL[dtype]      # values: before norm and rotation
    assert k_got[..., dim:].abs().sum() == 0 and v_got[..., dim:].abs().sum() == 0
    assert (kc == 9.0).sum() == kc.numel() - T * G * dp            # nothing else was written
    if not partials and dtype == torch.bfloat16:                   # many tokens: several heads per warp
        n = 1100
        big, bq = src.repeat(16, 1)[:n].contiguous(), torch.zeros(n, H * dp, dtype=dtype, device=dev)
        wide = torch.arange(1, 19, dtype=torch.int32, device=dev)[None]
        kb, vb = (torch.zeros(20, G, PAGE, dp, dtype=dtype, device=dev) for _ in range(2))
        bp = torch.arange(n, dtype=torch.int32, device=dev)
        cb, sb = K.rope_tables(n, rot, base, dev) if rot else (None, None)
        K.rotary_append(big, bq, 0, H * dp, H * dp, torch.zeros_like(bp), bp, cb, sb, wide, kb, vb, H, dim, rot, eps)
        br = big.view(n, H + G, dp)[..., :dim].double().cpu()
        want = O.rms(O.rotate(br, torch.arange(n), base, rot), eps)
        flat = lambda c: c[1:19].permute(0, 2, 1, 3).reshape(-1, G, dp)[:n]  # noqa: E731
        assert C.worst_row(bq.view(n, H, dp)[..., :dim].reshape(n, -1), want[:, :H].reshape(n, -1)) < TOL[dtype]
        assert C.worst_row(flat(kb)[..., :dim].reshape(n, -1), want[:, H:].reshape(n, -1)) < TOL[dtype]
        assert C.worst_row(flat(vb)[..., :dim].reshape(n, -1), br[:, H:].reshape(n, -1)) < 1e-6


# --------------------------------------------------------------------------- attention kernels
def _cache(seqs_k, seqs_v, dtype, dev, extra=3):
    """Scatter per-sequence keys / values [n, G, dp] over shuffled pages; unused entries hold large finite numbers."""
    G, dp = seqs_k[0].shape[1:]
    need = [-(-k.shape[0] // PAGE) for k in seqs_k]
    perm = (torch.randperm(sum(need) + extra, generator=torch.Generator().manual_seed(5)) + 1).tolist()
    n = len(perm) + 1
    kc, vc = torch.full((n, G, PAGE, dp), 50.0), torch.full((n, G, PAGE, dp), -50.0)
    table = torch.zeros(len(seqs_k), max(need) + 1, dtype=torch.int32)
    for b, (k, v) in enumerate(zip(seqs_k, seqs_v)):
        for j in range(need[b]):
            p = perm.pop()
            table[b, j] = p
            m = min(PAGE, k.shape[0] - j * PAGE)
            kc[p, :, :m], vc[p, :, :m] = (t[j * PAGE:j * PAGE + m].transpose(0, 1) for t in (k, v))
    return kc.to(dtype).to(dev), vc.to(dtype).to(dev), table.to(dev)


def _want(q, k, v, pos, window, scale, sink):
    mask = O.visible(k.shape[0], window or None)[pos.long()]
    return O.attend(q.double(), k.double(), v.double(), mask, scale, None if sink is None else sink.double()).reshape(len(pos), -1)


@pytest.mark.parametrize("kernel", ["rows f32", "rows bf16", "rows bf16 split", "prefill"])
@pytest.mark.parametrize("H,G,dim,window,sink", [(8, 2, 64, 0, True), (10, 2, 88, 112, True), (12, 1, 128, 200, False), (4, 4, 40, 64, True),
                                                 (3, 3, 24, 7, True), (20, 2, 80, 129, True), (9, 3, 48, 130, False), (2, 1, 200, 90, True), (2, 2, 256, 0, False)])
def test_chunked_attention_with_sink(cuda_device, kernel, H, G, dim, window, sink):
    """Portions that start anywhere, two requests of unequal length, every row against the oracle."""
    if kernel == "prefill" and dim > K.WINDOW_PREFILL_MAX_DIM:
        pytest.skip("the tensor-core prompt kernel covers heads up to 128")
    dtype = torch.float32 if kernel == "rows f32" else torch.bfloat16
    g = torch.Generator().manual_seed(dim + window)
    dev, scale = cuda_device, 1.5 / math.sqrt(dim)
    lens, starts = (417, 200), (150, 63)
    ks, vs = ([(torch.randn(n, G, dim, generator=g)).to(dtype).float() for n in lens] for _ in range(2))
    sk = 2 * torch.randn(H, generator=g) if sink else None
    kc, vc, table = _cache(ks, vs, dtype, dev)
    qs = [torch.randn(n - s, H, dim, generator=g).to(dtype) for n, s in zip(lens, starts)]
    q = torch.cat(qs).reshape(-1, H * dim).to(dev)
    pos = torch.cat([torch.arange(s, n) for n, s in zip(lens, starts)]).int()
    slot = torch.cat([torch.full((n - s,), b) for b, (n, s) in enumerate(zip(lens, starts))]).int().to(dev)
    want = torch.cat([_want(qq, k, v, torch.arange(s, n), window, scale, sk) for qq, k, v, n, s in zip(qs, ks, vs, lens, starts)])
    skd = None if sk is None else sk.to(dev)
    if kernel == "prefill":
        cu = torch.tensor([0, lens[0] - starts[0], q.shape[0]], dtype=torch.int32, device=dev)
        out = K.window_prefill(q, kc, vc, table, cu, pos.to(dev), slot, max(n - s for n, s in zip(lens, starts)), H, window=window, scale=scale,
                               sink=skd)
    else:
        ns = 3 if kernel.endswith("split") else 1
        scratch = torch.empty(max(1, K.rows_attn_scratch(q.shape[0], H, dim, ns)), device=dev)
        arrive = torch.zeros(q.shape[0] * H, dtype=torch.int32, device=dev)
        for _ in range(2):                               # the arrival counters must be back at zero for the second launch
            out = K.rows_attn(q, kc, vc, table, slot, pos.to(dev), H, window=window, scale=scale, sink=skd, nsplit=ns, scratch=scratch, arrive=arrive)
        assert arrive.abs().sum() == 0
        # a retired row (no keys) is zero, with lens given explicitly
        lens_t = (pos + 1).to(dev)
        lens_t[1] = 0
        o2 = K.rows_attn(q, kc, vc, table, slot, pos.to(dev), H, window=window, scale=scale, sink=skd, lens=lens_t)
        assert o2[1].abs().sum() == 0 and C.worst_relative_row(o2[2:], want[2:]) < ATTN[dtype]
    assert C.worst_relative_row(out, want) < ATTN[dtype]


@pytest.mark.parametrize("H,G", [(3, 3), (4, 1), (3, 1)])
@pytest.mark.parametrize("window,growing", [(0, False), (500, False), (512, True), (0, True)])
def test_long_prompt_portions(cuda_device, H, G, window, growing):
    """Many key tiles per row, two and more query tiles per portion; with ``growing`` the scores rise along the sequence, so
    the running maximum (and the accumulator) is rescaled again and again."""
    dev, dim, n, start, scale = cuda_device, 64, 1400, 333, 0.25
    g = torch.Generator().manual_seed(H + window)
    k, v = torch.randn(n, G, dim, generator=g), torch.randn(n, G, dim, generator=g)
    q = torch.randn(n - start, H, dim, generator=g)
    if growing:
        k[..., 0] = torch.linspace(0.0, 40.0, n)[:, None]
        q[..., 0] = 4.0
    k, v, q = k.bfloat16(), v.bfloat16(), q.bfloat16()
    kc, vc, table = _cache([k.float()], [v.float()], torch.bfloat16, dev)
    pos = torch.arange(start, n, dtype=torch.int32)
    sink = torch.randn(H, generator=g) if window else None
    want = _want(q, k, v, pos, window, scale, sink)
    out = K.window_prefill(q.reshape(len(pos), -1).to(dev), kc, vc, table, torch.tensor([0, n - start], dtype=torch.int32, device=dev), pos.to(dev),
                           torch.zeros(n - start, dtype=torch.int32, device=dev), n - start, H, window=window, scale=scale,
                           sink=None if sink is None else sink.to(dev))
    assert C.worst_relative_row(out, want) < ATTN[torch.bfloat16]


@pytest.mark.parametrize("kernel", ["rows", "prefill"])
@pytest.mark.parametrize("window", [64, 100, 256, 300])
def test_single_keys_at_chunk_and_page_edges(cuda_device, kernel, window):
    """One key stands out for the queries around it: just inside and just outside every chunk edge, at page borders, far
    back. The value behind it is the output wherever it is visible and absent one position further."""
    dev, H, G, dim, n = cuda_device, 4, 1, 64, 700
    g = torch.Generator().manual_seed(window)
    scale = 1.0 / 8
    spots = sorted({p for e in range(0, n, window) for p in (e - 1, e, e + 1, e + 63, e + 64) if 0 <= p < n} | {0, 1, 63, 64, 127, 128, n - 1})
    k = 0.1 * torch.randn(n, G, dim, generator=g)
    v = torch.randn(n, G, dim, generator=g)
    for spot in spots:
        kk = k.clone()
        kk[spot] = 0.0
        kk[spot, :, 0] = 12.0
        kc, vc, table = _cache([kk], [v], torch.bfloat16, dev)
        ends = sorted({p for p in (spot, spot + 1, (spot // window + 1) * window - 1, (spot // window + 1) * window, n - 1) if spot <= p < n})
        q = 0.1 * torch.randn(len(ends), H, dim, generator=g)
        q[..., 0] = 10.0                                  # score 15 for the key that stands out, near 0 for the others
        q = q.bfloat16()
        pos = torch.tensor(ends, dtype=torch.int32)
        want = _want(q, kk.bfloat16(), v.bfloat16(), pos, window, scale, None)
        qd, slot = q.reshape(len(ends), -1).to(dev), torch.zeros(len(ends), dtype=torch.int32, device=dev)
        if kernel == "rows":
            got = K.rows_attn(qd, kc, vc, table, slot, pos.to(dev), H, window=window, scale=scale)
        else:                                             # every row a portion of its own
            cu = torch.arange(len(ends) + 1, dtype=torch.int32, device=dev)
            got = K.window_prefill(qd, kc, vc, table, cu, pos.to(dev), slot, 1, H, window=window, scale=scale)
        assert C.worst_relative_row(got, want) < ATTN[torch.bfloat16], (spot, ends)
        seen = torch.tensor([p // window == spot // window for p in ends])
        near = (got.float().cpu().view(len(ends), H, dim) - v[spot].bfloat16().float()).norm(dim=-1).mean(-1)
        assert (near[seen] < 0.1).all() and (near[~seen] > 1.0).all()


def test_sink_counts_once_in_the_denominator(cuda_device):
    dev, dim = cuda_device, 32
    k = torch.zeros(130, 1, dim)
    v = torch.ones(130, 1, dim)
    kc, vc, table = _cache([k], [v], torch.bfloat16, dev)
    q = torch.zeros(130, 2 * dim, dtype=torch.bfloat16, device=dev)
    pos = torch.arange(130, dtype=torch.int32, device=dev)
    slot = torch.zeros(130, dtype=torch.int32, device=dev)
    sink = torch.tensor([math.log(3.0), -30.0], device=dev)
    want = torch.stack([torch.arange(1, 131) / (torch.arange(1, 131) + 3.0), torch.ones(130)], 1)      # n keys of weight 1 and a sink of weight 3
    cu = torch.tensor([0, 130], dtype=torch.int32, device=dev)
    scratch, arrive = torch.empty(K.rows_attn_scratch(130, 2, dim, 2), device=dev), torch.zeros(260, dtype=torch.int32, device=dev)
    for got in (K.window_prefill(q, kc, vc, table, cu, pos, slot, 130, 2, scale=0.7, sink=sink),
                K.rows_attn(q, kc, vc, table, slot, pos, 2, scale=0.7, sink=sink),
                K.rows_attn(q, kc, vc, table, slot, pos, 2, scale=0.7, sink=sink, nsplit=2, scratch=scratch, arrive=arrive)):
        assert (got.float().cpu().view(130, 2, dim) - want[..., None]).abs().max() < 2.5e-3


# --------------------------------------------------------------------------- mixture of experts
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,E,top,groups,ff,shared,width", [(1, 6, 3, (3, 2), 36, 50, 100), (37, 8, 2, (4, 1), 64, 0, 64), (300, 5, 5, (1, 1), 40, 40, 72),
                                                          (200, 64, 6, (8, 3), 32, 96, 128), (260, 1, 1, (1, 1), 200, 8, 264), (90, 300, 4, (10, 10), 16, 16, 48)])
def test_mixture(cuda_device, dtype, T, E, top, groups, ff, shared, width):
    from rpeg_b200.models.registry import config_from_hf
    from rpeg_b200.models.dulisun import DulisunModel
    cfg = C.config(width, 32, [C.layer(1, 1, 8, 1.0, mlp=C.moe(E, top, ff, groups, shared or None))])
    t = C.tensors(cfg, T + E)
    m = DulisunModel(config_from_hf(cfg), cuda_device, dtype=dtype, seed=None)
    m.p["l0.router"][:E, :width].copy_(t["l0.mlp.router"])
    for s in range(E):
        m.put_expert(0, s, t[f"l0.mlp.e{s}.up"].to(cuda_device), t[f"l0.mlp.e{s}.down"].to(cuda_device))
    if shared:
        m.put_shared(0, t["l0.mlp.shared.up"].to(cuda_device), t["l0.mlp.shared.down"].to(cuda_device))
    h = torch.randn(T, width, generator=torch.Generator().manual_seed(3)).bfloat16()
    td = {n: v.double() for n, v in t.items()}
    want = O.moe(h.double(), td, "l0.mlp.", cfg["layers"][0]["mlp"])
    hd = _pad(h.to(dtype), m.cfg.width_p).to(cuda_device)
    w = torch.zeros(m.cfg.width_p, dtype=dtype, device=cuda_device)
    for decode in ((False, True) if T <= 256 and dtype == torch.bfloat16 else (False,)):
        counts = torch.zeros(E, dtype=torch.int32, device=cuda_device)
        out = m._mixture(0, m.cfg.layers[0].mlp, hd, counts, decode)
        assert int(counts.sum()) == T * top
        # the routing itself: scores of the chosen experts, not renormalised
        s = torch.softmax(h.double() @ td["l0.mlp.router"].T, -1)
        ids = [O.route(r.tolist(), cfg["layers"][0]["mlp"]["router"]) for r in s]
        got_w = torch.sort(out.weights.double().cpu(), dim=1, descending=True).values
        assert (got_w - torch.stack([r[i] for r, i in zip(s, ids)])).abs().max() < 1e-5
        x = torch.zeros(T, m.cfg.width_p, device=cuda_device)
        K.residual_norm(out, w, 1e-3, width, x=x)
        assert C.worst_row(x[:, :width], O.rms(want, 1e-3)) < 3 * TOL[dtype]
        assert x[:, width:].abs().sum() == 0


def test_router_groups_and_ties(cuda_device):
    """The group with the single best expert wins over groups with better seconds; equal scores go to the lower number."""
    z = torch.full((4, 12), -3.0)
    z[0, 11], z[0, 0], z[0, 1], z[0, 2] = 2.0, 1.9, 1.8, 1.7           # 3 groups of 4: group 2 holds the best
    z[1] = 0.0                                                          # all equal
    z[2, 5], z[2, 9] = 1.0, 1.0                                         # groups 1 and 2 tie
    z[3, 3], z[3, 7], z[3, 10] = 3.0, 2.0, 1.0
    def run(keep, top):
        counts = torch.zeros(12, dtype=torch.int32, device=cuda_device)
        ids, wts, ticket = K.moe_route(z.to(cuda_device), 12, top, counts, n_groups=3, keep_groups=keep)
        assert torch.equal(counts.cpu(), torch.bincount(ids.cpu().flatten().long(), minlength=12).int())
        return ids.cpu().tolist(), wts.cpu()
    ids, wts = run(1, 2)
    assert ids[0][0] == 11 and ids[0][1] == 8 and ids[1] == [0, 1] and ids[2] == [5, 4] and ids[3] == [3, 0]
    assert torch.allclose(wts[0, 0], torch.softmax(z[0], -1)[11])
    assert run(2, 3)[0][3] == [3, 7, 0] and run(3, 3)[0][3] == [3, 7, 10] and run(2, 8)[0][1] == list(range(8))
    _, w = K.moe_route(z.to(cuda_device), 12, 3, torch.zeros(12, dtype=torch.int32, device=cuda_device), renormalize=True)[:2]
    assert torch.allclose(w.sum(1).cpu(), torch.ones(4))


def test_gemm_f32(cuda_device):
    g = torch.Generator().manual_seed(0)
    for M, N, Kd in ((1, 8, 5), (70, 130, 200), (129, 64, 1000)):
        a, b = torch.randn(M, Kd, generator=g).to(cuda_device), torch.randn(N, Kd, generator=g).to(cuda_device)
        assert C.rel(K.gemm_f32(a, b), a.double() @ b.double().T) < 1e-6


# --------------------------------------------------------------------------- the model
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(config, fp64 tensors, directory, {dtype: model}) per case, built once."""
    made = {}

    def get(name):
        if name not in made:
            cfg = {"unlike": C.unlike, "regular": C.regular, "long": C.long_chunks}[name]()
            t = C.tensors(cfg, 11)
            path = C.write(cfg, t, tmp_path_factory.mktemp(name) / "model")
            made[name] = (cfg, t, path, {d: load_model(path, "cuda:0", dtype=d) for d in DT})
        return made[name]

    return get


def _tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _session(model, max_tokens=768, slots=8, pages=None):
    budget = (pages or slots * (max_tokens // PAGE) + 1) * page_elems(model.kv_geometry()) * model.dtype.itemsize
    return Session(Generator(model, max_slots=slots, max_seq_len=max_tokens, kv_budget_bytes=budget, use_graphs=False))


def _feed(s, rid, tokens, sizes):
    """All logits of one request fed in portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        out.append(s.feed([(rid, tokens[at:at + n], list(range(n)))])[0].float())
        at, i = at + n, i + 1
    return torch.cat(out)


def _close(got, want, dtype):
    """fp32: every row. bf16: rounding turns over the closest routing decisions (and the keys of such a token reach the next
    few), so all but a few rows, and those few stay bounded."""
    e = C.row_errors(got, want)
    if dtype == torch.float32:
        assert e.max() < 5e-5
    else:
        assert e.quantile(0.5) < 2e-2 and e.quantile(0.93) < 8e-2 and e.max() < 1.5


@pytest.mark.parametrize("name,n", [("unlike", 260), ("regular", 200), ("long", 420)])
def test_prefill_decode_and_portions_match_the_oracle(models, name, n):
    cfg, t, _, ms = models(name)
    tokens = _tokens(cfg, n, 1)
    layers = []
    want = O.forward(cfg, t, tokens, layers)
    for dtype, model in ms.items():
        trace = []
        dev_tok = torch.tensor(tokens, dtype=torch.int32, device="cuda")
        xf, _ = model.forward(dev_tok, torch.arange(n, dtype=torch.int32, device="cuda"), torch.tensor([0, n], dtype=torch.int32, device="cuda"), n,
                              trace=trace)
        for a, b in zip(trace, layers):
            _close(a, b, dtype)
        _close(model.lm_logits(xf), want, dtype)
        s = _session(model)
        for sizes in ([n], [1], [n - 40, 1], [64], [2], [3, 61, 65, 2, 1, 1, 30, 7]):
            if dtype == torch.bfloat16 and sizes == [2]:
                sizes = [2] * 20 + [n]
            _close(_feed(s, "r", tokens, sizes), want, dtype)
            s.end("r")                                    # the next pass runs on used pages
        assert s.gen.pool.available() == s.gen.pool.num_pages - 1


@pytest.mark.parametrize("name", ["unlike", "regular"])
def test_first_tokens(models, name):
    cfg, t, _, ms = models(name)
    for n in (1, 2, 3):
        tokens = _tokens(cfg, n, 40 + n)
        want = O.forward(cfg, t, tokens)
        s = _session(ms[torch.float32])
        assert C.worst_row(_feed(s, "a", tokens, [n]), want) < 5e-5 and C.worst_row(_feed(s, "b", tokens, [1]), want) < 5e-5


def test_mixed_batches_match_each_request_alone(models):
    """Unequal requests, prompts and single tokens in one step, requests that come and go; against each one alone."""
    cfg, t, _, ms = models("unlike")
    model = ms[torch.float32]
    seqs = {f"q{i}": _tokens(cfg, n, 60 + i) for i, n in enumerate((150, 67, 1, 200, 33, 129))}
    want = {k: O.forward(cfg, t, v) for k, v in seqs.items()}
    s = _session(model, 256, 4, pages=4 * 4 + 1)
    g = torch.Generator().manual_seed(8)
    waiting, live, done, got = list(seqs), [], {k: 0 for k in seqs}, {k: [] for k in seqs}
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step = []
        for k in live:
            n = min(len(seqs[k]) - done[k], int((1, 1, 1, 2, 5, 40, 70)[int(torch.randint(0, 7, (1,), generator=g))]))
            step.append((k, seqs[k][done[k]:done[k] + n], list(range(n))))
            done[k] += n
        for (k, _, _), out in zip(step, s.feed(step)):
            got[k].append(out)
        for k in [k for k in live if done[k] == len(seqs[k])]:
            assert C.worst_row(torch.cat(got[k]), want[k]) < 5e-5, k
            s.end(k)
            live.remove(k)
    assert s.gen.pool.available() == s.gen.pool.num_pages - 1


def test_pages_behind_the_chunk_are_given_back_and_used_again(models):
    """With chunks everywhere a request holds only its current chunk's pages; what it gave back serves others meanwhile."""
    cfg, t, _, ms = models("regular")
    model = ms[torch.float32]
    a, b = _tokens(cfg, 300, 5), _tokens(cfg, 300, 6)
    s = _session(model, 320, 4, pages=8)                  # two requests of 300 tokens need 10 pages at once
    got = {"a": [], "b": []}
    for i in range(0, 300, 20):
        for k, v in (("a", a), ("b", b)):
            got[k].append(s.feed([(k, v[i:i + 20], list(range(20)))])[0])
    for k, v in (("a", a), ("b", b)):
        assert C.worst_row(torch.cat(got[k]), O.forward(cfg, t, v)) < 5e-5
        assert s.requests[k].gone == 270 // PAGE
        s.end(k)
    assert s.gen.pool.available() == s.gen.pool.num_pages - 1


def _greedy_ok(cfg, t, prompt, generated, tol):
    """Every generated token is the oracle's choice, or one within ``tol`` (relative to the logits' spread) of it."""
    logits = O.forward(cfg, t, prompt + generated)[len(prompt) - 1:-1]
    spread = logits.std(-1)
    picked = logits.gather(1, torch.tensor(generated)[:, None])[:, 0]
    return bool((logits.max(-1).values - picked <= tol * spread).all())


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name,portion", [("unlike", 0), ("regular", 37)])
def test_greedy_generation(models, dtype, name, portion):
    """The framework's own scheduler: more rows than slots, graphs, prompts in portions, rows that end early, a long decode
    over several chunk edges."""
    cfg, t, _, ms = models(name)
    model = ms[dtype]
    prompts = [_tokens(cfg, n, 80 + n) for n in (1, 30, 89, 90, 91, 140)]
    new = 120
    gen = Generator(model, max_slots=4, max_seq_len=320, kv_budget_bytes=1e9, eos_id=-1, sync_interval=4, prefill_portion=portion)
    res = gen.generate([torch.tensor(p, dtype=torch.int32) for p in prompts], new, greedy=True, forced_lens=None)
    assert res.lengths.tolist() == [new] * len(prompts)
    for p, row in zip(prompts, res.tokens.tolist()):
        assert _greedy_ok(cfg, t, p, row, 1e-4 if dtype == torch.float32 else 0.1)
    if name == "regular":
        assert res.counters["kv_pages_passed"] > 0
    assert res.counters["kv_pages_taken"] == res.counters["kv_pages_returned"] and gen.pool.available() == gen.pool.num_pages - 1
    # log-probs of the sampling policy agree with the packed forward over the finished rows
    for p, row, lp in list(zip(prompts, res.tokens, res.logprobs))[2:4]:
        ro = A.Rollout(torch.tensor([p], dtype=torch.int32, device="cuda"), [len(p)], row[None], [new], lp[None], torch.ones(1, new, device="cuda"))
        again = A.sequence_logprobs(model, ro, A.AlgoConfig(micro_tokens=4096, head_chunk=64))
        assert (again[0] - lp).abs().max() < (1e-3 if dtype == torch.float32 else 0.15)


def test_generation_with_few_pages_and_shared_prompts(models):
    """Preemption, prompt pages shared by a group of samples, and page release together: greedy rows stay what they are."""
    cfg, t, _, ms = models("regular")
    model = ms[torch.float32]
    uniq = [_tokens(cfg, n, 200 + n) for n in (130, 64)]
    for prompt in uniq:
        rows = [torch.tensor(prompt, dtype=torch.int32)] * 4
        page_bytes = page_elems(model.kv_geometry()) * 4
        tight = Generator(model, max_slots=4, max_seq_len=300, kv_budget_bytes=8.5 * page_bytes, eos_id=-1, sync_interval=4, use_graphs=False)
        res = tight.generate(rows, 100, greedy=True, group_size=4)
        for row in res.tokens.tolist():
            assert _greedy_ok(cfg, t, prompt, row, 1e-4)
        assert tight.pool.available() == tight.pool.num_pages - 1
    # a cache carved from a buffer full of other bits
    gen = Generator(ms[torch.bfloat16], max_slots=2, max_seq_len=256, kv_storage=torch.full((page_elems(model.kv_geometry()) * 12,), float("nan"),
                    dtype=torch.bfloat16, device="cuda"), eos_id=-1, sync_interval=4)
    row = gen.generate([torch.tensor(uniq[0], dtype=torch.int32)], 20, greedy=True).tokens[0].tolist()
    assert _greedy_ok(cfg, t, uniq[0], row, 0.1)


def test_sampling_filters_work_on_this_family(models):
    cfg, t, _, ms = models("regular")
    for dtype in DT:
        gen = Generator(ms[dtype], max_slots=2, max_seq_len=128, kv_budget_bytes=1e8, eos_id=-1, sync_interval=4)
        p = [torch.tensor(_tokens(cfg, 20, 3), dtype=torch.int32)]
        a, b = gen.generate(p, 24, greedy=True), gen.generate(p, 24, seed=3, top_k=1)
        assert torch.equal(a.tokens, b.tokens) or dtype == torch.bfloat16
        c = gen.generate(p, 24, seed=4, temperature=0.7, top_p=0.5)
        assert int(c.tokens.max()) < cfg["vocab"] and (c.logprobs <= 0).all()


def test_checked_mode_covers_the_family(models):
    cfg, _, _, ms = models("unlike")
    prev = checked.set_enabled(True)
    try:
        for model in ms.values():
            s = _session(model, 128, 2)
            _feed(s, "a", _tokens(cfg, 90, 2), [70, 1, 1, 10])
            s.gen.page_table[s.requests["a"].slot, 1] = 10 ** 6
            with pytest.raises(checked.KernelArgumentError):
                s.feed([("a", [1], [])])
    finally:
        checked.set_enabled(prev)


# --------------------------------------------------------------------------- other models and command lines
def test_session_drives_the_llama_family_too(cuda_device):
    """A model without cached prefill: portions behind a prefix go through the decode step one token at a time."""
    from rpeg_b200.models.llama import LlamaConfig, LlamaModel
    cfg = LlamaConfig.tiny(n_layers=2)
    model = LlamaModel(cfg, cuda_device, seed=6)
    tokens = torch.randint(0, cfg.vocab, (150,), generator=torch.Generator().manual_seed(1)).tolist()
    s = Session(Generator(model, max_slots=4, max_seq_len=256, kv_budget_bytes=1e8, use_graphs=False))
    whole = _feed(s, "w", tokens, [150])
    for sizes in ([100, 1], [60, 7, 1, 40]):
        got = _feed(s, "p", tokens, sizes)
        s.end("p")
        assert C.worst_row(got, whole) < 5e-2


def test_generate_command(models, capsys):
    from rpeg_b200.engine import generate
    cfg, t, path, _ = models("regular")
    p = _tokens(cfg, 50, 9)
    assert generate.main(["--model", str(path), "--dtype", "float32", "--prompt", ",".join(map(str, p)), "--prompt", "5", "--max-new", "30",
                          "--greedy", "--prefill-portion", "16"]) == 0
    rows = [json.loads(line) for line in capsys.readouterr().out.splitlines() if line.startswith("{")]
    assert [r["row"] for r in rows] == [0, 1] and all(len(r["tokens"]) == 30 for r in rows)
    assert _greedy_ok(cfg, t, p, rows[0]["tokens"], 1e-4) and _greedy_ok(cfg, t, [5], rows[1]["tokens"], 1e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_command(models, tmp_path, dtype):
    import numpy as np
    cfg, t, path, _ = models("unlike")
    a, b = _tokens(cfg, 140, 21), _tokens(cfg, 20, 22)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:100], "want": [0, 49, 50, 99]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[100:102], "want": []}, {"id": "b", "tokens": b, "want": [19]}], "end": ["b"]}]
    steps += [{"step": 2 + i, "entries": [{"id": "a", "tokens": [tok], "want": [0]}], "end": ["a"] if i == 37 else []} for i, tok in enumerate(a[102:])]
    run = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(path), "--dtype", dtype, "--out", str(tmp_path),
                          "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [ln for ln in run.stdout.splitlines() if ln.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    read = lambda i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])  # noqa: E731
    want = torch.cat([O.forward(cfg, t, a)[[0, 49, 50, 99] + list(range(102, 140))], O.forward(cfg, t, b)[[19]]])
    _close(torch.cat([read(0)] + [read(2 + i) for i in range(38)] + [read(1)]), want, getattr(torch, dtype))
