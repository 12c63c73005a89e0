"""GPU tests of the Zafopel family against the plain oracle: every mechanism alone, then the model through the generator's
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

import dulisun_cases as D  # noqa: E402
import zafopel_cases as C  # noqa: E402
import zafopel_oracle as O  # noqa: E402
from rpeg_b200.engine import algorithms as A  # noqa: E402
from rpeg_b200.engine.generation import PAGE, Generator, page_elems  # noqa: E402
from rpeg_b200.engine.session import Session  # noqa: E402
from rpeg_b200.models.registry import config_from_hf, load_model  # noqa: E402
from rpeg_b200.models.zafopel import ZafopelModel  # noqa: E402
from rpeg_b200.ops import checked  # noqa: E402
from rpeg_b200.ops import kernels as K  # noqa: E402

DT = (torch.float32, torch.bfloat16)
TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}
ATTN = {torch.float32: 2e-5, torch.bfloat16: 6e-3}        # scores, weights and sums are fp32: only the output is rounded
ROOT = Path(__file__).resolve().parent.parent


@pytest.fixture(autouse=True)
def _status():
    yield
    K.check_status()


def _pad(x, n):
    return torch.nn.functional.pad(x, (0, n - x.shape[-1])).contiguous()


def _p8(n):
    return -(-n // 8) * 8


# --------------------------------------------------------------------------- stream and norm
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("rows,d,alpha", [(1, 5, 0.5), (3, 100, -1.75), (37, 256, 0.03), (5, 1030, 4.0)])
def test_stream_update(cuda_device, dtype, rows, d, alpha):
    g = torch.Generator().manual_seed(d)
    dev, dp = cuda_device, _p8(d)
    w, b = (_pad((0.5 * torch.randn(d, generator=g)).to(dtype), dp).to(dev) for _ in range(2))
    t = {"n": w[:d].double().cpu(), "n.b": b[:d].double().cpu(), "n.alpha": torch.tensor(alpha, dtype=torch.float64)}
    al = torch.tensor(alpha, device=dev)
    x0 = _pad(torch.randn(rows, d, generator=g) * torch.logspace(-4, 1, d), dp).to(dev)

    def act():
        return _pad(torch.randn(rows, d, generator=g).to(dtype), dp).to(dev)

    def parts(n):
        buf = torch.zeros(n, rows, dp, device=dev)
        buf[..., :d] = torch.randn(n, rows, d, generator=g).to(dev)
        return K.Partials(buf.view(-1), n, rows, dp), buf.double().sum(0).cpu()

    def check(a, b_src, add, **kw):
        x = x0.clone()
        y = K.stream_update(a, b_src, al, w, b, x, **kw)
        want = add if kw else x0.double().cpu() + add
        assert D.rel(x, want) < 1e-6 and x[:, d:].abs().sum() == 0
        # the norm alone, on the stream as the kernel wrote it
        norm = O.dynamic_tanh(x[:, :d].double().cpu(), t, "n")
        assert ((y[:, :d].double().cpu() - norm).abs() <= (2e-7 if dtype == torch.float32 else 5e-3) * (norm.abs() + t["n"].abs() + t["n.b"].abs()) + 1e-12).all()
        assert y[:, d:].abs().sum() == 0

    a, a2 = act(), act()
    check(a, None, a.double().cpu())
    check(a, a2, a.double().cpu() + a2.double().cpu())
    top, E = 3, 7
    row_of = torch.randperm(rows * top, generator=g).int().view(rows, top).to(dev)
    ys = _pad(torch.randn(rows * top, d, generator=g).to(dtype), dp).to(dev)
    wts = torch.rand(rows, top, generator=g).to(dev)
    plain = ys.double().cpu()[row_of.cpu().long()].sum(1)
    weighed = (ys.double().cpu()[row_of.cpu().long()] * wts.double().cpu()[..., None]).sum(1)
    check(a, K.MoEOutput(ys, row_of, None, 0), a.double().cpu() + plain)
    check(a, K.MoEOutput(ys, row_of, wts, 0), a.double().cpu() + weighed)
    table = _pad(torch.randn(9, d, generator=g).to(dtype), dp).to(dev)
    ids = torch.randint(0, 9, (rows,), generator=g, dtype=torch.int32).to(dev)
    check(table, None, table[ids.long()].double().cpu(), ids=ids)
    if dtype == torch.bfloat16:
        (p1, s1), (p2, s2) = parts(3), parts(1)
        check(p1, None, s1)
        check(p1, p2, s1 + s2)
        check(p2, K.MoEOutput(ys, row_of, None, 0), s2 + plain)


def test_tanh_is_accurate_over_its_range(cuda_device):
    """Small arguments in relative terms, the switch between the two forms, saturation."""
    z = torch.cat([torch.logspace(-20, 2, 6000), torch.linspace(0.4, 0.7, 1992)])
    z = torch.cat([z, -z]).view(-1, 8)
    x = z.to(cuda_device).clone()
    one, zero = torch.ones(8, device=cuda_device), torch.zeros(8, device=cuda_device)
    y = K.stream_update(torch.zeros_like(x), None, torch.tensor(1.0, device=cuda_device), one, zero, x).double().cpu()
    want = torch.tanh(z.double())
    assert ((y - want).abs() / want.abs()).max() < 6e-7 and y.abs().max() == 1.0


# --------------------------------------------------------------------------- latents, rotations, per-head products
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("partials", [False, True])
@pytest.mark.parametrize("H,dim,rot,rank,nq", [(5, 20, 12, 36, 44), (3, 48, 32, 88, 0), (1, 8, 2, 200, 1500), (4, 40, 0, 24, 8)])
def test_latent_rows(cuda_device, dtype, partials, H, dim, rot, rank, nq):
    if partials and dtype == torch.float32:
        pytest.skip("split-K partials belong to the bf16 path")
    g = torch.Generator().manual_seed(dim + rank)
    dev, T, eps, base = cuda_device, 70, 1e-2, 300.0
    dp, rp, kp, qp = _p8(dim), _p8(rot), _p8(rank), _p8(nq)
    widths = [(nq, qp), (rank, kp), (rot, rp)] + [(dim, dp), (rot, rp)] * H
    cols = [_pad(torch.randn(3 if partials else 1, T, n, generator=g), p) for n, p in widths]
    raw = torch.cat(cols, -1)
    if partials:
        src = K.Partials(raw.reshape(-1).to(dev), 3, T, raw.shape[-1])
        raw = raw.double().sum(0)
    else:
        raw = raw[0].to(dtype)
        src = raw.to(dev)
        raw = raw.double()
    slot = torch.tensor([0] * 40 + [1] * 30, dtype=torch.int32)
    pos = torch.cat([torch.arange(100, 140), torch.arange(3, 33)]).int()
    table = torch.tensor([[5, 2, 7], [1, 4, 0]], dtype=torch.int32)
    cache = torch.full((8, 1, PAGE, kp + rp), 9.0, dtype=dtype, device=dev)
    cos_t, sin_t = K.rope_tables(256, rot, base, dev) if rot else (None, None)
    kw, kn = _pad((1 + torch.rand(nq or 8, generator=g)).to(dtype), qp or 8).to(dev), _pad((1 + torch.rand(rank, generator=g)).to(dtype), kp).to(dev)
    cq = torch.zeros(T, qp or 8, dtype=dtype, device=dev)
    nope = torch.zeros(T, H * dp, dtype=dtype, device=dev)
    wide = torch.full((T, H, kp + rp), 3.0, dtype=dtype, device=dev)
    c0 = qp + kp + rp
    args = (pos.to(dev), slot.to(dev), cos_t, sin_t, rot, rp, eps)
    K.latent_rows(src, *args, q_latent=(0, nq, kw, cq) if nq else None, kv=(qp, rank, kn, cache, table.to(dev)), queries=(c0, H, dp, nope, wide[:, :, kp:]))
    rotated = lambda x: O.rotate(x, pos, base) if rot else x  # noqa: E731
    if nq:
        assert D.worst_row(cq[:, :nq], O.rms(raw[:, :nq], kw[:nq].double().cpu(), eps)) < TOL[dtype] and cq[:, nq:].abs().sum() == 0
    got = cache[table[slot.long(), pos.long() // PAGE].long(), 0, pos.long() % PAGE]
    assert D.worst_row(got[:, :rank], O.rms(raw[:, qp:qp + rank], kn[:rank].double().cpu(), eps)) < TOL[dtype]
    if rot:
        assert D.worst_row(got[:, kp:kp + rot], rotated(raw[:, qp + kp:qp + kp + rot])) < TOL[dtype]
    assert got[:, rank:kp].abs().sum() == 0 and got[:, kp + rot:].abs().sum() == 0
    assert (cache == 9.0).sum() == cache.numel() - T * (kp + rp)              # nothing else was written
    q = raw[:, c0:].view(T, H, dp + rp)
    assert D.worst_row(nope.view(T, -1), q[:, :, :dp].reshape(T, -1)) < TOL[dtype] and (wide[:, :, :kp] == 3.0).all()
    if rot:
        assert D.worst_row(wide[:, :, kp:kp + rot].reshape(T, -1), rotated(q[:, :, dp:dp + rot]).reshape(T, -1)) < TOL[dtype]
        assert wide[:, :, kp + rot:].abs().sum() == 0
    if not partials:                                                          # queries alone, rotated where they are
        view = src[:, c0:].unflatten(1, (H, dp + rp))
        before = src.clone()
        K.latent_rows(src, *args, queries=(c0, H, dp, None, view[:, :, dp:]))
        assert torch.equal(view[:, :, dp:].contiguous(), wide[:, :, kp:].contiguous()) and torch.equal(src[:, :c0], before[:, :c0])
        assert torch.equal(view[:, :, :dp].contiguous(), before[:, c0:].unflatten(1, (H, dp + rp))[:, :, :dp].contiguous())


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,H,N,Kd", [(1, 3, 8, 40), (70, 5, 136, 24), (300, 2, 512, 128), (33, 17, 128, 512), (129, 64, 200, 72)])
def test_head_gemm(cuda_device, dtype, T, H, N, Kd):
    g = torch.Generator().manual_seed(N)
    a = torch.randn(T, H, Kd + 16, generator=g).to(dtype).to(cuda_device)[:, :, 8:8 + Kd]          # strided views on both sides
    for transposed in (False, True):
        w = (torch.randn(H, Kd, N, generator=g) if transposed else torch.randn(H, N, Kd, generator=g)).to(dtype).to(cuda_device) / math.sqrt(Kd)
        buf = torch.full((T, H, N + 24), 7.0, dtype=dtype, device=cuda_device)
        K.head_gemm(a, w, buf[:, :, 16:16 + N], transposed=transposed)
        want = torch.einsum("thk,hkn->thn" if transposed else "thk,hnk->thn", a.double(), w.double())
        assert D.worst_row(buf[:, :, 16:16 + N].reshape(T, -1), want.reshape(T, -1)) < (1e-5 if dtype == torch.float32 else 5e-3)
        assert (buf[:, :, :16] == 7.0).all() and (buf[:, :, 16 + N:] == 7.0).all()


# --------------------------------------------------------------------------- attention kernels
def _cache(seqs, dtype, dev, extra=3):
    """Scatter cached rows [n, W] of every sequence over shuffled pages; unused entries hold large finite numbers."""
    W = seqs[0].shape[1]
    need = [-(-s.shape[0] // PAGE) for s in seqs]
    perm = (torch.randperm(sum(need) + extra, generator=torch.Generator().manual_seed(5)) + 1).tolist()
    c = torch.full((len(perm) + 1, 1, PAGE, W), 50.0)
    table = torch.zeros(len(seqs), max(need) + 1, dtype=torch.int32)
    for b, s in enumerate(seqs):
        for j in range(need[b]):
            p = perm.pop()
            table[b, j] = p
            part = s[j * PAGE:(j + 1) * PAGE]
            c[p, 0, : part.shape[0]] = part
    return c.to(dtype).to(dev), table.to(dev)


def _want(q, rows, rank, pos, window, scale, sink):
    """Averaged latents [T, H * rank]: every head's key is the cached row."""
    n, H = rows.shape[0], q.shape[1]
    k = rows.double()[:, None].expand(n, H, rows.shape[1])
    mask = O.visible(n, window or None)[pos.long()]
    return O.attend(q.double(), k, k[..., :rank], mask, scale, None if sink is None else sink.double()).reshape(len(pos), -1)


def _score(kernel, q, cache, rank, table, slot, pos, window, scale, sink, lens=None):
    if kernel.startswith("rows"):
        return K.latent_attn_rows(q, cache, rank, table, slot, pos, window=window, scale=scale, sink=sink, lens=lens)
    ns = 5 if kernel.endswith("split") else 1
    scratch = torch.full((max(1, K.latent_decode_scratch(q.shape[0], q.shape[1], rank, ns)),), float("nan"), device=q.device)
    return K.latent_decode(q, cache, rank, table, slot, pos, window=window, scale=scale, sink=sink, lens=lens, nsplit=ns, scratch=scratch)


@pytest.mark.parametrize("kernel", ["rows f32", "rows bf16", "tensor", "tensor split"])
@pytest.mark.parametrize("H,rank,W,window,sink", [(7, 88, 112, 0, True), (5, 40, 56, 37, False), (33, 512, 576, 0, True), (32, 512, 576, 64, False), (70, 136, 144, 65, True),
                                                  (1, 8, 8, 1, False), (16, 320, 384, 200, True), (3, 256, 288, 2, True), (9, 64, 576, 300, False)])
def test_scores_on_cached_rows(cuda_device, kernel, H, rank, W, window, sink):
    """Query rows that stand anywhere, of two requests of unequal length, every row against the oracle."""
    dtype = torch.float32 if kernel == "rows f32" else torch.bfloat16
    g = torch.Generator().manual_seed(rank + window)
    dev, scale = cuda_device, 1.5 / math.sqrt(W)
    lens = (417, 200)
    seqs = [torch.randn(n, W, generator=g).to(dtype).float() for n in lens]
    pos = [torch.cat([torch.arange(0, 3), torch.arange(60, 68), torch.arange(125, 131), torch.arange(n - 9, n)]).int() for n in lens]
    qs = [torch.randn(len(p), H, W, generator=g).to(dtype) for p in pos]
    sk = 2 * torch.randn(H, generator=g) if sink else None
    cache, table = _cache(seqs, dtype, dev)
    want = torch.cat([_want(q, s, rank, p, window, scale, sk) for q, s, p in zip(qs, seqs, pos)])
    q, p = torch.cat(qs).to(dev), torch.cat(pos).to(dev)
    slot = torch.cat([torch.full((len(x),), b) for b, x in enumerate(pos)]).int().to(dev)
    skd = None if sk is None else sk.to(dev)
    out = _score(kernel, q, cache, rank, table, slot, p, window, scale, skd)
    assert D.worst_relative_row(out.reshape(len(p), -1), want) < ATTN[dtype]
    lens_t = p + 1                                           # a retired row (no keys) is zero, with lens given explicitly
    lens_t[1] = 0
    out = _score(kernel, q, cache, rank, table, slot, torch.zeros_like(p), window, scale, skd, lens_t).reshape(len(p), -1)
    assert out[1].abs().sum() == 0 and D.worst_relative_row(out[2:], want[2:]) < ATTN[dtype]


@pytest.mark.parametrize("kernel", ["rows bf16", "tensor", "tensor split"])
@pytest.mark.parametrize("falling", [False, True])
def test_growing_scores_rescale_the_accumulator(cuda_device, kernel, falling):
    """Scores that rise along the sequence for some heads and fall for others, by far more than the lazy rescaling allows."""
    g = torch.Generator().manual_seed(3)
    H, rank, W, n, scale = 12, 256, 320, 900, 0.2
    rows = torch.randn(n, W, generator=g)
    rows[:, 0] = torch.linspace(40.0, 0.0, n) if falling else torch.linspace(0.0, 40.0, n)
    q = torch.randn(7, H, W, generator=g)
    q[:, ::2, 0], q[:, 1::2, 0] = 6.0, -6.0
    rows, q = rows.bfloat16(), q.bfloat16()
    cache, table = _cache([rows.float()], torch.bfloat16, cuda_device)
    pos = torch.arange(n - 7, n).int()
    out = _score(kernel, q.to(cuda_device), cache, rank, table, torch.zeros(7, dtype=torch.int32, device=cuda_device), pos.to(cuda_device), 0, scale, None)
    assert D.worst_relative_row(out.reshape(7, -1), _want(q, rows, rank, pos, 0, scale, None)) < ATTN[torch.bfloat16]


def _formed(rows, rank, H, dim, vdim, g, dtype=torch.bfloat16):
    """Key and value maps and what they make of the rows, as the product lays them out."""
    uk, uv = (torch.randn(H, n, rank, generator=g) / math.sqrt(rank) for n in (dim, vdim))
    k, v = (torch.einsum("nr,hdr->nhd", rows[:, :rank].double(), w.double()).to(dtype) for w in (uk, uv))
    return k, v


def _prefill(cuda_device, lens, starts, H, dim, rot, vdim, window, scale, sink, g, tweak=None, portion_rows=None):
    """Run ``latent_prefill`` on portions ``starts[b] .. lens[b]`` of random sequences; (result, wanted) ``[T, H * vdim]``."""
    dev, rank = cuda_device, 64
    dp, rp, vp = _p8(dim), _p8(rot), _p8(vdim)
    bf = torch.bfloat16
    qs, ks, vs, wants, kvs, gathered, off, lo = [], [], [], [], [], [], [0], []
    for n, s in zip(lens, starts):
        rows = torch.randn(n, rank + rot, generator=g).to(bf)
        q = torch.randn(n - s, H, dim + rot, generator=g).to(bf)
        k, v = _formed(rows, rank, H, dim, vdim, g)
        if tweak is not None:
            tweak(q, k, v, rows)
        full_k = torch.cat([k, rows[:, None, rank:].expand(n, H, rot)], -1)
        wants.append(O.attend(q.double(), full_k.double(), v.double(), O.visible(n, window or None)[s:n], scale, None if sink is None else sink.double()).reshape(n - s, -1))
        first = max(0, s - window + 1) if window else 0
        qs.append(torch.cat([_pad(q[..., :dim], dp), _pad(q[..., dim:], rp)], -1))
        kvs.append(torch.cat([_pad(k[first:], dp).reshape(n - first, -1), _pad(v[first:], vp).reshape(n - first, -1)], 1))
        gathered.append(torch.cat([rows[first:, :rank], _pad(rows[first:, rank:], rp)], 1))
        lo.append(first)
        off.append(off[-1] + n - first)
    cu = torch.tensor([0] + [n - s for n, s in zip(lens, starts)]).cumsum(0).int().to(dev)
    pos = torch.cat([torch.arange(s, n) for n, s in zip(lens, starts)]).int().to(dev)
    out = K.latent_prefill(torch.cat(qs).to(dev), torch.cat(kvs).contiguous().to(dev), torch.cat(gathered).contiguous().to(dev), dp, vp, rank, cu, pos,
                           torch.tensor(off, dtype=torch.int32, device=dev), torch.tensor(lo, dtype=torch.int32, device=dev), max(n - s for n, s in zip(lens, starts)),
                           window=window, scale=scale, sink=None if sink is None else sink.to(dev))
    T = int(cu[-1])
    return out.view(T, H, vp)[..., :vdim].reshape(T, -1), torch.cat(wants)


@pytest.mark.parametrize("H,dim,rot,vdim,window,sink", [(5, 56, 24, 56, 0, True), (2, 20, 12, 28, 37, False), (3, 128, 64, 128, 0, True), (1, 128, 64, 96, 200, True), (2, 40, 2, 72, 1, False),
                                                        (2, 72, 16, 16, 64, True), (1, 192, 0, 128, 129, False), (2, 64, 128, 64, 5, True), (4, 8, 8, 8, 300, False)])
def test_prompt_attention_on_formed_keys(cuda_device, H, dim, rot, vdim, window, sink):
    g = torch.Generator().manual_seed(dim + window)
    sk = 2 * torch.randn(H, generator=g) if sink else None
    got, want = _prefill(cuda_device, (417, 200, 130), (150, 63, 0), H, dim, rot, vdim, window, 1.5 / math.sqrt(dim + rot), sk, g)
    assert D.worst_relative_row(got, want) < ATTN[torch.bfloat16]


@pytest.mark.parametrize("window,start", [(0, 0), (500, 333), (512, 0), (100, 700)])
@pytest.mark.parametrize("growing", [False, True])
def test_long_prompts(cuda_device, window, start, growing):
    """Many key tiles and several pairs of query tiles; with ``growing`` the scores rise, so the accumulator is rescaled again and again."""
    g = torch.Generator().manual_seed(window)

    def tweak(q, k, v, rows):
        if growing:
            k[..., 0] = torch.linspace(0.0, 40.0, k.shape[0])[:, None].bfloat16()
            q[..., 0] = 4.0

    got, want = _prefill(cuda_device, (1400,), (start,), 2, 64, 32, 64, window, 0.2, torch.randn(2, generator=g) if window else None, g, tweak)
    assert D.worst_relative_row(got, want) < ATTN[torch.bfloat16]


@pytest.mark.parametrize("kernel", ["rows f32", "rows bf16", "tensor", "tensor split", "formed"])
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 200])
def test_single_keys_at_window_and_page_edges(cuda_device, kernel, window):
    """One key stands out for the queries around it: visible up to ``window - 1`` positions on, gone one further, at page borders and at the
    start of the sequence. The latent behind it is the output wherever it is visible."""
    dtype = torch.float32 if kernel == "rows f32" else torch.bfloat16
    dev, H, rank, W, n, scale = cuda_device, 4, 64, 80, 500, 1.0 / 8
    g = torch.Generator().manual_seed(window)
    base = 0.1 * torch.randn(n, W, generator=g)
    for spot in (0, 1, 63, 64, 127, 128, 200, 255, 256):
        rows = base.clone()
        rows[spot] = torch.randn(W, generator=g)
        rows[spot, 64:] = 0.0
        rows[spot, 64] = 12.0                                # in the rotated part: it decides the score, not the value
        rows = rows.to(dtype)
        ends = sorted({p for p in (spot, spot + 1, spot + window - 1, spot + window, spot + window + 1) if spot <= p < n})
        q = 0.1 * torch.randn(len(ends), H, W, generator=g)
        q[..., 64] = 12.0
        q = q.to(dtype)
        pos = torch.tensor(ends, dtype=torch.int32)
        want = _want(q, rows, rank, pos, window, scale, None)
        if kernel == "formed":                               # every row a portion of its own; keys and values are the latents themselves
            lo = [max(0, p - window + 1) for p in ends]
            seen_rows = torch.cat([rows[a:p + 1] for a, p in zip(lo, ends)])
            off = torch.tensor([0] + [p + 1 - a for a, p in zip(lo, ends)]).cumsum(0).int().to(dev)
            kv = torch.cat([seen_rows[:, None, :rank].expand(-1, H, rank).reshape(len(seen_rows), -1)] * 2, 1).contiguous()
            got = K.latent_prefill(q.to(dev), kv.to(dev), seen_rows.contiguous().to(dev), rank, rank, rank, torch.arange(len(ends) + 1, dtype=torch.int32, device=dev),
                                   pos.to(dev), off, torch.tensor(lo, dtype=torch.int32, device=dev), 1, window=window, scale=scale)
        else:
            cache, table = _cache([rows.float()], dtype, dev)
            got = _score(kernel, q.to(dev), cache, rank, table, torch.zeros(len(ends), dtype=torch.int32, device=dev), pos.to(dev), window, scale, None)
        got = got.reshape(len(ends), -1)
        assert D.worst_relative_row(got, want) < 2 * ATTN[dtype], (spot, ends)
        seen = torch.tensor([p - spot < window for p in ends])
        near = (got.float().cpu().view(len(ends), H, rank) - rows[spot, :rank].float()).norm(dim=-1).mean(-1)
        assert (near[seen] < 0.2).all() and (near[~seen] > 3.0).all(), (spot, near)


def test_sink_counts_once_in_the_denominator(cuda_device):
    dev, rank, n = cuda_device, 32, 130
    rows = torch.zeros(n, 48)
    rows[:, :rank] = 1.0
    cache, table = _cache([rows], torch.bfloat16, dev)
    c32, t32 = _cache([rows], torch.float32, dev)
    q = torch.zeros(n, 2, 48, dtype=torch.bfloat16, device=dev)
    pos, slot = torch.arange(n, dtype=torch.int32, device=dev), torch.zeros(n, dtype=torch.int32, device=dev)
    sink = torch.tensor([math.log(3.0), -30.0], device=dev)
    want = torch.stack([torch.arange(1, n + 1) / (torch.arange(1, n + 1) + 3.0), torch.ones(n)], 1)[..., None]   # n keys of weight 1, a sink of weight 3
    for kernel in ("rows f32", "rows bf16", "tensor", "tensor split"):
        f32 = kernel == "rows f32"
        got = _score(kernel, q.float() if f32 else q, c32 if f32 else cache, rank, t32 if f32 else table, slot, pos, 0, 0.7, sink)
        assert (got.float().cpu() - want).abs().max() < 2.5e-3
    i32 = dict(dtype=torch.int32, device=dev)
    kv = torch.ones(n, 2 * 2 * 32, dtype=torch.bfloat16, device=dev)
    got = K.latent_prefill(q, kv, rows.bfloat16().to(dev), 32, 32, 32, torch.tensor([0, n], **i32), pos, torch.tensor([0, n], **i32), torch.zeros(1, **i32), n, scale=0.7, sink=sink)
    assert (got.float().cpu().view(n, 2, 32) - want).abs().max() < 2.5e-3


@pytest.mark.parametrize("dtype", DT)
def test_latent_gather(cuda_device, dtype):
    g = torch.Generator().manual_seed(1)
    seqs = [torch.randn(n, 40, generator=g).to(dtype).float() for n in (200, 65, 131)]
    cache, table = _cache(seqs, dtype, cuda_device)
    slot = torch.tensor([2, 2, 0, 1, 1], dtype=torch.int32, device=cuda_device)              # requests on table rows 2, 0, 1
    cu = torch.tensor([0, 2, 3, 5], dtype=torch.int32, device=cuda_device)
    want = torch.cat([seqs[2][60:130], seqs[0][130:195], seqs[1][:3]])
    off = torch.tensor([0, 70, 135, 138], dtype=torch.int32, device=cuda_device)
    got = K.latent_gather(cache, table, slot, cu, off, torch.tensor([60, 130, 0], dtype=torch.int32, device=cuda_device), 138)
    assert torch.equal(got.float().cpu(), want)


# --------------------------------------------------------------------------- feed-forwards
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,E,top,ff,width", [(1, 6, 3, 36, 100), (37, 7, 1, 88, 64), (300, 5, 5, 40, 72), (200, 64, 6, 32, 128), (260, 1, 1, 200, 264), (90, 300, 4, 16, 48)])
def test_mixture_with_scaled_inputs(cuda_device, dtype, T, E, top, ff, width):
    cfg = C.config(width, 32, [C.layer(1, 8, 2, 8, 8, 1.0, 100.0, window=4, mlp=C.moe(E, top, ff))])
    t = C.tensors(cfg, T + E)
    m = ZafopelModel(config_from_hf(cfg), cuda_device, dtype=dtype, seed=None)
    m.put_router(0, t["l0.mlp.router"])
    for s in range(E):
        m.put_expert(0, s, *(t[f"l0.mlp.e{s}.{n}"].to(cuda_device) for n in ("gate", "up", "down")))
    h = torch.randn(T, width, generator=torch.Generator().manual_seed(3)).bfloat16()
    td = {n: v.double() for n, v in t.items()}
    want = O.moe(h.double(), td, "l0.mlp.", cfg["layers"][0]["mlp"])
    scores, chosen = O.route(h.double(), td, "l0.mlp.", cfg["layers"][0]["mlp"]["router"])
    hd = _pad(h.to(dtype), m.cfg.width_p).to(cuda_device)
    mx = m.cfg.layers[0].mixer
    router = m._ff_rows(0)
    logits = [m._lin(hd, router, False, f32_out=True)]
    if T <= 256 and dtype == torch.bfloat16:                 # decode: the router's columns of the stacked projection's partials
        logits.append(m._lin(hd, m.p["l0.w_in"], True).columns(mx.q_in + mx.kv_in))
    for z in logits:
        counts = torch.zeros(E, dtype=torch.int32, device=cuda_device)
        ids, wts, ticket = K.moe_route(z, E, top, counts, sigmoid=True)
        assert int(counts.sum()) == T * top
        got_w = torch.sort(wts.double().cpu(), dim=1, descending=True).values
        assert (got_w - torch.stack([s[i] for s, i in zip(scores, chosen)])).abs().max() < 1e-5      # sigmoid scores, not renormalised
        counts.zero_()
        out = m._feed_forward(0, hd, z, counts, False)
        assert out.weights is None
        x = torch.zeros(T, m.cfg.width_p, device=cuda_device)
        one = torch.ones(m.cfg.width_p, dtype=dtype, device=cuda_device)
        K.stream_update(torch.zeros(T, m.cfg.width_p, dtype=dtype, device=cuda_device), out, torch.tensor(1.0, device=cuda_device), one, one, x)
        assert D.worst_row(x[:, :width], want) < TOL[dtype] and x[:, width:].abs().sum() == 0


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,ff,width", [(1, 50, 100), (130, 264, 64), (40, 1000, 136), (300, 24, 1030)])
def test_dense_feed_forward(cuda_device, dtype, T, ff, width):
    cfg = C.config(width, 32, [C.layer(1, 8, 2, 8, 8, 1.0, 100.0, window=4, mlp=C.dense(ff))])
    t = C.tensors(cfg, ff)
    m = ZafopelModel(config_from_hf(cfg), cuda_device, dtype=dtype, seed=None)
    m.put_dense(0, t["l0.mlp.up"], t["l0.mlp.down"])
    h = torch.randn(T, width, generator=torch.Generator().manual_seed(3)).bfloat16()
    want = O.dense(h.double(), {n: v.double() for n, v in t.items()}, "l0.mlp.")
    hd = _pad(h.to(dtype), m.cfg.width_p).to(cuda_device)
    mx, fp = m.cfg.layers[0].mixer, _p8(ff)
    for decode in ((False, True) if dtype == torch.bfloat16 and T <= 256 else (False,)):
        first = None
        if decode or dtype == torch.float32:                 # the first product comes with the layer's projection
            first = torch.full((T, fp), 5.0, dtype=dtype, device=cuda_device)
            K.latent_rows(m._lin(hd, m.p["l0.w_in"], decode), torch.zeros(T, dtype=torch.int32, device=cuda_device), torch.zeros(T, dtype=torch.int32, device=cuda_device),
                          None, None, 0, 8, 1e-5, ff=(mx.q_in + mx.kv_in, first))
            assert D.worst_row(first[:, :ff], torch.relu(h.double() @ t["l0.mlp.up"].double().T) ** 2) < TOL[dtype] and first[:, ff:].abs().sum() == 0
        out = m._feed_forward(0, hd, first, None, decode)
        out = out.reduce() if isinstance(out, K.Partials) else out
        assert D.worst_row(out[:, :width], want) < TOL[dtype] and out[:, width:].abs().sum() == 0


# --------------------------------------------------------------------------- the model
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(config, tensors, directory, {dtype: model}) per case, built once."""
    made = {}

    def get(name):
        if name not in made:
            cfg = getattr(C, name)()
            t = C.tensors(cfg, 11)
            path = D.write(cfg, t, tmp_path_factory.mktemp(name) / "model")
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
    """fp32: every row. bf16: rounding turns over the closest routing decisions (and later tokens see such a token), so all but a few
    rows, and those few stay bounded."""
    e = D.row_errors(got, want)
    if dtype == torch.float32:
        assert e.max() < 5e-5
    else:
        assert e.quantile(0.5) < 2e-2 and e.quantile(0.93) < 8e-2 and e.max() < 1.5


@pytest.mark.parametrize("name,n", [("unlike", 260), ("sliding", 230), ("wide", 300)])
@pytest.mark.parametrize("way", ["chosen", "formed", "scored", "cuda cores"])
def test_prefill_decode_and_portions_match_the_oracle(models, name, n, way, monkeypatch):
    cfg, t, _, ms = models(name)
    tokens = _tokens(cfg, n, 1)
    layers = []
    want = O.forward(cfg, t, tokens, layers)
    for dtype, model in ms.items():
        if dtype == torch.float32 and way != "chosen":
            continue
        if way == "formed":                                   # wherever the kernel takes the head sizes
            monkeypatch.setattr(model, "_forms_keys", lambda m, spans: K.latent_prefill_fits(m.dim_p, m.rot_p, m.vdim_p))
        elif way != "chosen":
            monkeypatch.setattr(model, "_forms_keys", lambda m, spans: False)
        if way == "cuda cores":
            monkeypatch.setattr(K, "latent_decode_fits", lambda *a: False)
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
            s.end("r")                                        # the next pass runs on used pages
        assert s.gen.pool.available() == s.gen.pool.num_pages - 1


@pytest.mark.parametrize("name", ["unlike", "sliding"])
def test_first_tokens(models, name):
    cfg, t, _, ms = models(name)
    for n in (1, 2, 3):
        tokens = _tokens(cfg, n, 40 + n)
        want = O.forward(cfg, t, tokens)
        s = _session(ms[torch.float32])
        assert D.worst_row(_feed(s, "a", tokens, [n]), want) < 5e-5 and D.worst_row(_feed(s, "b", tokens, [1]), want) < 5e-5
        _close(_feed(_session(ms[torch.bfloat16]), "a", tokens, [n]), want, torch.bfloat16)


def test_far_token_and_sinks_decide_the_logits(models, tmp_path):
    """One far token that stands out among hundreds of equal ones, sinks as heavy as all of them together, a layer that reads the other's
    latents: whatever is left out moves the logits by four orders of magnitude more than the tolerance."""
    cfg = C.config(32, 64, [C.layer(2, 16, 8, 16, 24, 1.0, 1e4, q_rank=16), C.layer(2, 16, 8, 16, 24, 1.0, 1e4, q_rank=16, kv_from=0)])
    t = C.tensors(cfg, 7)
    for i in range(2):
        t[f"l{i}.mix.sink"] = torch.tensor([14.0, 12.0]).bfloat16()
    n = 400
    tokens = [56] + [11] * (n - 1)
    want = O.forward(cfg, t, tokens)
    without = [O.forward(cfg, {**t, f"l{i}.mix.sink": t[f"l{i}.mix.sink"] - 9}, tokens) for i in range(2)] + [O.forward(cfg, t, [11] * n)]
    assert all(D.worst_row(w[-3:], want[-3:]) > 0.3 for w in without)
    path = D.write(cfg, t, tmp_path / "m")
    for dtype in DT:
        m = load_model(path, "cuda:0", dtype=dtype)
        for sizes in ([n - 3, 1], [n], [130, 2]):
            _close(_feed(_session(m), "a", tokens, sizes), want, dtype)


def test_mixed_batches_match_each_request_alone(models):
    """Unequal requests, prompts and single tokens in one step, requests that come and go; against each one alone."""
    cfg, t, _, ms = models("unlike")
    for dtype, model in ms.items():
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
                _close(torch.cat(got[k]), want[k], dtype)
                s.end(k)
                live.remove(k)
        assert s.gen.pool.available() == s.gen.pool.num_pages - 1


def test_pages_behind_the_windows_are_given_back_and_used_again(models):
    """With windows everywhere a request holds only the pages its windows touch; what it gave back serves others meanwhile."""
    cfg, t, _, ms = models("sliding")
    for dtype, model in ms.items():
        a, b = _tokens(cfg, 300, 5), _tokens(cfg, 300, 6)
        s = _session(model, 320, 4, pages=8)                  # two requests of 300 tokens need 10 pages at once
        got = {"a": [], "b": []}
        for i in range(0, 300, 20):
            for k, v in (("a", a), ("b", b)):
                got[k].append(s.feed([(k, v[i:i + 20], list(range(20)))])[0])
        for k, v in (("a", a), ("b", b)):
            _close(torch.cat(got[k]), O.forward(cfg, t, v), dtype)
            assert s.requests[k].gone == (300 - 89) // PAGE
            s.end(k)
        assert s.gen.pool.available() == s.gen.pool.num_pages - 1


def _greedy_ok(cfg, t, prompt, generated, tol):
    """Every generated token is the oracle's choice, or one within ``tol`` (relative to the logits' spread) of it."""
    logits = O.forward(cfg, t, prompt + generated)[len(prompt) - 1:-1]
    spread = logits.std(-1)
    picked = logits.gather(1, torch.tensor(generated)[:, None])[:, 0]
    return ((logits.max(-1).values - picked) / spread <= tol).double().mean().item()


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name,portion", [("unlike", 0), ("sliding", 37)])
def test_greedy_generation(models, dtype, name, portion):
    """The framework's own scheduler: more rows than slots, graphs, prompts in portions, a long decode over several windows."""
    cfg, t, _, ms = models(name)
    model = ms[dtype]
    prompts = [_tokens(cfg, n, 80 + n) for n in (1, 30, 89, 90, 91, 140)]
    new = 120
    gen = Generator(model, max_slots=4, max_seq_len=320, kv_budget_bytes=1e9, eos_id=-1, sync_interval=4, prefill_portion=portion)
    res = gen.generate([torch.tensor(p, dtype=torch.int32) for p in prompts], new, greedy=True)
    assert res.lengths.tolist() == [new] * len(prompts)
    for p, row in zip(prompts, res.tokens.tolist()):          # bf16: a routing decision may turn over, which moves a row's logits for a while
        assert _greedy_ok(cfg, t, p, row, 1e-4 if dtype == torch.float32 else 0.15) >= (1.0 if dtype == torch.float32 else 0.9)
    if name == "sliding":
        assert res.counters["kv_pages_passed"] > 0
    assert res.counters["kv_pages_taken"] == res.counters["kv_pages_returned"] and gen.pool.available() == gen.pool.num_pages - 1
    # log-probs of the sampling policy agree with the packed forward over the finished rows
    for p, row, lp in list(zip(prompts, res.tokens, res.logprobs))[2:4]:
        ro = A.Rollout(torch.tensor([p], dtype=torch.int32, device="cuda"), [len(p)], row[None], [new], lp[None], torch.ones(1, new, device="cuda"))
        again = A.sequence_logprobs(model, ro, A.AlgoConfig(micro_tokens=4096, head_chunk=64))
        d = (again[0] - lp).abs()
        assert d.max() < 1e-3 if dtype == torch.float32 else d.quantile(0.9) < 0.1


def test_generation_with_few_pages_and_shared_prompts(models):
    """Preemption, prompt pages shared by a group of samples, and page release together: greedy rows stay what they are."""
    cfg, t, _, ms = models("sliding")
    model = ms[torch.float32]
    uniq = [_tokens(cfg, n, 200 + n) for n in (130, 64)]
    for prompt in uniq:
        rows = [torch.tensor(prompt, dtype=torch.int32)] * 4
        page_bytes = page_elems(model.kv_geometry()) * 4
        tight = Generator(model, max_slots=4, max_seq_len=300, kv_budget_bytes=8.5 * page_bytes, eos_id=-1, sync_interval=4, use_graphs=False)
        res = tight.generate(rows, 100, greedy=True, group_size=4)
        for row in res.tokens.tolist():
            assert _greedy_ok(cfg, t, prompt, row, 1e-4) == 1.0
        assert tight.pool.available() == tight.pool.num_pages - 1
    # a cache carved from a buffer full of other bits
    gen = Generator(ms[torch.bfloat16], max_slots=2, max_seq_len=256, kv_storage=torch.full((page_elems(model.kv_geometry()) * 12,), float("nan"),
                    dtype=torch.bfloat16, device="cuda"), eos_id=-1, sync_interval=4)
    row = gen.generate([torch.tensor(uniq[0], dtype=torch.int32)], 20, greedy=True).tokens[0].tolist()
    assert _greedy_ok(cfg, t, uniq[0], row, 0.15) >= 0.9


def test_decode_with_many_splits(models):
    """One row over a long cache: its pages are shared by many CTAs, window edges fall inside splits."""
    cfg, t, _, ms = models("wide")
    n = 700
    tokens = _tokens(cfg, n, 77)
    want = O.forward(cfg, t, tokens)[n - 6:]
    for dtype, model in ms.items():
        s = _session(model, 768, 2)
        s.feed([("r", tokens[: n - 6], [])])
        got = torch.cat([s.feed([("r", [tok], [0])])[0].float() for tok in tokens[n - 6:]])
        assert model._nsplit(model.cfg.layers[0].mixer, 1, 12) > 1 if dtype == torch.bfloat16 else True
        _close(got, want, dtype)


def test_sampling_filters_work_on_this_family(models):
    cfg, t, _, ms = models("sliding")
    for dtype in DT:
        gen = Generator(ms[dtype], max_slots=2, max_seq_len=128, kv_budget_bytes=1e8, eos_id=-1, sync_interval=4)
        p = [torch.tensor(_tokens(cfg, 20, 3), dtype=torch.int32)]
        a, b = gen.generate(p, 24, greedy=True), gen.generate(p, 24, seed=3, top_k=1)
        assert torch.equal(a.tokens, b.tokens) or dtype == torch.bfloat16
        c = gen.generate(p, 24, seed=4, temperature=0.7, top_p=0.5)
        assert int(c.tokens.max()) < cfg["vocab"] and (c.logprobs <= 0).all()


def test_checked_mode_covers_the_family(models, monkeypatch):
    cfg, _, _, ms = models("unlike")
    prev = checked.set_enabled(True)
    try:
        for model in ms.values():
            for way in (True, False):
                if way:
                    monkeypatch.setattr(model, "_forms_keys", lambda m, spans: not model.f32 and K.latent_prefill_fits(m.dim_p, m.rot_p, m.vdim_p))
                s = _session(model, 128, 2)
                _feed(s, "a", _tokens(cfg, 90, 2), [70, 1, 1, 10])
                s.gen.page_table[s.requests["a"].slot, 1] = 10 ** 6
                for portion in ([1], [1, 2, 3, 4]):
                    with pytest.raises(checked.KernelArgumentError):
                        s.feed([("a", portion, [])])
                monkeypatch.undo()
    finally:
        checked.set_enabled(prev)


# --------------------------------------------------------------------------- command lines
def test_generate_command(models, capsys):
    from rpeg_b200.engine import generate
    cfg, t, path, _ = models("sliding")
    p = _tokens(cfg, 50, 9)
    assert generate.main(["--model", str(path), "--dtype", "float32", "--prompt", ",".join(map(str, p)), "--prompt", "5", "--max-new", "30",
                          "--greedy", "--prefill-portion", "16"]) == 0
    rows = [json.loads(line) for line in capsys.readouterr().out.splitlines() if line.startswith("{")]
    assert [r["row"] for r in rows] == [0, 1] and all(len(r["tokens"]) == 30 for r in rows)
    assert _greedy_ok(cfg, t, p, rows[0]["tokens"], 1e-4) == 1.0 and _greedy_ok(cfg, t, [5], rows[1]["tokens"], 1e-4) == 1.0


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
