"""Zafopel decoder: latent attention (sliding or causal with a softmax sink; a layer may read an earlier layer's latents) beside a
feed-forward (dense squared relu, or a sigmoid-routed mixture whose weights scale the experts' inputs), both fed by one elementwise norm.
Every layer has its own sizes.

    x = E[token]
    h = tanh(alpha x) * w + b                         one norm per layer, no statistics
    x += mixer(h) + ff(h)
    logits = H (tanh(alpha x) * w + b)

    latent row of a token      [ rms(D h) | rotated part ]              all that is cached
    head i                     k = [U_i c | rotated part], v = V_i c, q from h directly or through a latent of its own

What runs where:
  * stream, norms, angles, scores, softmax, routing are fp32; the matrix products take bf16 operands and accumulate in fp32
    (``dtype=torch.float32`` runs everything in true fp32);
  * one projection per layer gives the query side, the latent and (decode) the router logits or a dense feed-forward's first
    product; one kernel then normalises, rotates, takes the activation and writes the latents into the cache (``ops.kernels.latent_rows``);
  * decoded tokens and short portions never form keys or values: queries go through U_i transposed and score the cached rows, and
    the averaged latents go through V_i (``head_gemm`` before and after the attention). Longer portions gather the rows they see, form
    keys and values with one GEMM and run an ordinary tensor-core attention over them. ``_forms_keys`` picks the cheaper way;
  * one kernel per layer updates the stream from both sublayers' outputs and applies the next norm (``ops.kernels.stream_update``).

This family is served (generation, log-probs); it has no backward pass here.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, Iterable, List, Optional, Tuple, Union

import torch

from ..ops import kernels as K
from .llama import FlatLayout
from .served import ServedDecoder, pad8


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int                            # unrotated query / key dimensions of a head
    rot_dim: int                        # rotated ones; the key's are shared by all heads
    vdim: int
    kv_rank: int                        # latent width
    scale: float
    rot_base: float = 10000.0
    q_rank: int = 0                     # width of the query latent; 0: queries come straight from the input
    window: int = 0                     # keys are visible up to this many positions back, the own one included; 0: all earlier keys
    sink: bool = False
    kv_from: Optional[int] = None       # layer whose latents this one reads instead of its own

    @property
    def dim_p(self) -> int:
        return pad8(self.dim)

    @property
    def rot_p(self) -> int:
        return pad8(self.rot_dim)

    @property
    def vdim_p(self) -> int:
        return pad8(self.vdim)

    @property
    def rank_p(self) -> int:
        return pad8(self.kv_rank)

    @property
    def q_rank_p(self) -> int:
        return pad8(self.q_rank)

    @property
    def head_width(self) -> int:
        return self.dim_p + self.rot_p

    @property
    def q_width(self) -> int:
        return self.heads * self.head_width

    @property
    def row_width(self) -> int:
        """Elements of a cached row."""
        return self.rank_p + self.rot_p

    @property
    def q_in(self) -> int:
        """Rows of the layer's input projection that belong to the queries."""
        return self.q_rank_p if self.q_rank else self.q_width

    @property
    def kv_in(self) -> int:
        return self.row_width if self.kv_from is None else 0


@dataclass(frozen=True)
class DenseFF:
    ff: int

    @property
    def ff_p(self) -> int:
        return pad8(self.ff)

    @property
    def in_p(self) -> int:
        return self.ff_p


@dataclass(frozen=True)
class InputScaledMixture:
    """Gated experts; a choice's sigmoid score multiplies the expert's input."""
    experts: int
    top: int
    ff: int

    @property
    def ff_p(self) -> int:
        return pad8(self.ff)

    @property
    def in_p(self) -> int:
        return pad8(self.experts)


@dataclass(frozen=True)
class ParallelLayer:
    mixer: LatentMixer
    mlp: Optional[Union[DenseFF, InputScaledMixture]] = None

    @property
    def ff_in(self) -> int:
        """Rows of the layer's input projection that belong to the feed-forward: the router, or a dense one's first product."""
        return 0 if self.mlp is None else self.mlp.in_p


@dataclass(frozen=True)
class ZafopelConfig:
    width: int
    vocab: int
    layers: Tuple[ParallelLayer, ...]
    norm_eps: float = 1e-6              # of the RMS norms on the latents
    max_pos: int = 4096                 # initial size of the rotary tables (they grow with the generator's row length)
    family: str = "zafopel"

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def d_model(self) -> int:
        return self.width

    @property
    def width_p(self) -> int:
        return pad8(self.width)

    @property
    def vocab_p(self) -> int:
        return pad8(self.vocab)

    def kv_geometry(self, tp: int = 1) -> List[Tuple[int, int, int]]:
        """(KV heads, key width, value width) of every layer's cache: one latent row per token, nothing for a layer that reads another's."""
        if tp != 1:
            raise ValueError("this family has no tensor-parallel cache layout")
        return [(1, l.mixer.row_width, 0) if l.mixer.kv_from is None else (0, 0, 0) for l in self.layers]

    def n_params(self) -> int:
        return ZafopelLayout(self).total


class ZafopelLayout(FlatLayout):
    """Flat offsets of every matrix (padded shapes)."""

    def __init__(self, cfg: ZafopelConfig):
        super().__init__()
        d = cfg.width_p
        self.add("embed", cfg.vocab_p, d)
        for i, layer in enumerate(cfg.layers):
            m, e = layer.mixer, layer.mlp
            self.add(f"l{i}.norm1", d)
            self.add(f"l{i}.norm1.b", d)
            self.add(f"l{i}.w_in", m.q_in + m.kv_in + layer.ff_in, d)          # queries (or their latent), latent and rotated part, router or dense up
            if m.q_rank:
                self.add(f"l{i}.q_norm", m.q_rank_p)
                self.add(f"l{i}.w_uq", m.q_width, m.q_rank_p)
            if m.kv_from is None:
                self.add(f"l{i}.kv_norm", m.rank_p)
            self.add(f"l{i}.w_ukv", m.heads * (m.dim_p + m.vdim_p), m.rank_p)  # key maps of all heads, then value maps
            self.add(f"l{i}.wo", d, m.heads * m.vdim_p)
            if isinstance(e, DenseFF):
                self.add(f"l{i}.w_down", d, e.ff_p)
            elif e is not None:
                self.add(f"l{i}.w_gate_up", e.experts, 2 * e.ff_p, d)
                self.add(f"l{i}.w_down", e.experts, d, e.ff_p)
        self.add("final_norm", d)
        self.add("final_norm.b", d)
        self.add("head", cfg.vocab_p, d)


class _Spans:
    """What the packed requests of one prefill see, per window: total rows, their offsets and first positions (host and device)."""

    def __init__(self, starts: List[int], lens: List[int], device):
        self.starts, self.lens, self.device = starts, lens, device
        self._made: Dict[int, tuple] = {}

    def total(self, window: int) -> int:
        return sum(n + (min(s, window - 1) if window else s) for s, n in zip(self.starts, self.lens))

    def pairs(self, window: int) -> float:
        """(query, visible key) pairs."""
        out = 0.0
        for s, n in zip(self.starts, self.lens):
            full = n * s + n * (n + 1) / 2
            cut = max(0, s + n - window) if window else 0          # queries that see less than everything before them
            first = max(s, window) if window else 0
            if cut:
                m = s + n - first
                full -= m * (first - window + 1) + m * (m - 1) / 2
            out += full
        return out

    def rows(self, window: int):
        """(total, offsets [B + 1], first visible positions [B]) on the device."""
        if window not in self._made:
            lo = [max(0, s - window + 1) if window else 0 for s in self.starts]
            off = [0]
            for s, n, l in zip(self.starts, self.lens, lo):
                off.append(off[-1] + s + n - l)
            both = torch.tensor(off + lo, dtype=torch.int32).to(self.device)
            self._made[window] = (off[-1], both[: len(off)], both[len(off):])
        return self._made[window]


class ZafopelModel(ServedDecoder):
    """Weights and kernels of one model on one GPU."""

    prefill_spans = True
    KERNEL_SOURCES = ("gemm.cu", "generate.cu", "loss.cu", "stream_update.cu", "latent.cu", "latent_decode.cu", "latent_prefill.cu", "head_gemm.cu",
                      "moe.cu", "gemm_f32.cu")

    def __init__(self, cfg: ZafopelConfig, device, *, dtype: torch.dtype = torch.bfloat16, seed: Optional[int] = 0, trainable: bool = False):
        """``seed=None`` leaves the weights zero (a checkpoint is about to be loaded)."""
        super().__init__(cfg, ZafopelLayout(cfg), device, dtype=dtype, trainable=trainable)
        f32 = dict(dtype=torch.float32, device=self.device)
        self.sink = [torch.zeros(l.mixer.heads, **f32) if l.mixer.sink else None for l in cfg.layers]
        self.alpha = torch.ones(cfg.n_layers + 1, **f32)           # per layer, then the last norm's
        self.max_experts = max([l.mlp.experts for l in cfg.layers if isinstance(l.mlp, InputScaledMixture)], default=1)
        self._split: Dict[Tuple[int, int], torch.Tensor] = {}
        if seed is not None:
            self.init_weights(seed)

    # ------------------------------------------------------------------ weights
    def init_weights(self, seed: int = 0) -> None:
        """Random weights of the true sizes (the padding stays zero), unit-gain matrices and norms near one."""
        gen = torch.Generator(device=self.device)
        gen.manual_seed(seed)

        def rnd(*shape: int) -> torch.Tensor:
            return torch.randn(shape, generator=gen, device=self.device, dtype=torch.float32)

        def lin(rows: int, cols: int) -> torch.Tensor:
            return rnd(rows, cols) / math.sqrt(cols)

        d = self.cfg.width
        self.p["embed"][: self.cfg.vocab, :d].copy_(rnd(self.cfg.vocab, d))
        self.p["head"][: self.cfg.vocab, :d].copy_(lin(self.cfg.vocab, d))
        self.put_norm(self.cfg.n_layers, torch.tensor(0.5), 1 + 0.1 * rnd(d), 0.1 * rnd(d))
        for i, layer in enumerate(self.cfg.layers):
            m, e = layer.mixer, layer.mlp
            self.put_norm(i, torch.tensor(0.5), 1 + 0.1 * rnd(d), 0.1 * rnd(d))
            if m.q_rank:
                self.put_query_latent(i, lin(m.q_rank, d), 1 + 0.1 * rnd(m.q_rank))
            self.put_q(i, lin(m.heads * (m.dim + m.rot_dim), m.q_rank or d))
            if m.kv_from is None:
                self.put_latent(i, lin(m.kv_rank + m.rot_dim, d), 1 + 0.1 * rnd(m.kv_rank))
            self.put_kv_maps(i, lin(m.heads * m.dim, m.kv_rank), lin(m.heads * m.vdim, m.kv_rank))
            self.put_o(i, lin(d, m.heads * m.vdim))
            if m.sink:
                self.sink[i].copy_(rnd(m.heads))
            if isinstance(e, DenseFF):
                self.put_dense(i, lin(e.ff, d), lin(d, e.ff))
            elif e is not None:
                self.put_router(i, lin(e.experts, d))
                for s in range(e.experts):
                    self.put_expert(i, s, lin(e.ff, d), lin(e.ff, d), lin(d, e.ff))

    def put_norm(self, i: int, alpha: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> None:
        """Norm of layer ``i`` (``n_layers``: the last one)."""
        name = "final_norm" if i == self.cfg.n_layers else f"l{i}.norm1"
        self.alpha[i] = alpha.float().to(self.device)
        self.p[name][: self.cfg.width].copy_(w)
        self.p[name + ".b"][: self.cfg.width].copy_(b)

    def put_query_latent(self, i: int, dq: torch.Tensor, norm: torch.Tensor) -> None:
        r = self.cfg.layers[i].mixer.q_rank
        self.p[f"l{i}.w_in"][:r, : self.cfg.width].copy_(dq)
        self.p[f"l{i}.q_norm"][:r].copy_(norm)

    def put_q(self, i: int, wq: torch.Tensor) -> None:
        """``[heads * (dim + rot_dim), q_rank or width]``; both parts of a head are padded."""
        m = self.cfg.layers[i].mixer
        dst = (self.p[f"l{i}.w_uq"] if m.q_rank else self.p[f"l{i}.w_in"][: m.q_width]).view(m.heads, m.head_width, -1)
        src = wq.view(m.heads, m.dim + m.rot_dim, -1)
        n = src.shape[2]
        dst[:, : m.dim, :n].copy_(src[:, : m.dim])
        dst[:, m.dim_p:m.dim_p + m.rot_dim, :n].copy_(src[:, m.dim:])

    def put_latent(self, i: int, dkv: torch.Tensor, norm: torch.Tensor) -> None:
        m, d = self.cfg.layers[i].mixer, self.cfg.width
        dst = self.p[f"l{i}.w_in"][m.q_in:m.q_in + m.kv_in]
        dst[: m.kv_rank, :d].copy_(dkv[: m.kv_rank])
        dst[m.rank_p:m.rank_p + m.rot_dim, :d].copy_(dkv[m.kv_rank:])
        self.p[f"l{i}.kv_norm"][: m.kv_rank].copy_(norm)

    def put_kv_maps(self, i: int, uk: torch.Tensor, uv: torch.Tensor) -> None:
        m = self.cfg.layers[i].mixer
        k, v = self._kv_maps(i)
        k[:, : m.dim, : m.kv_rank].copy_(uk.view(m.heads, m.dim, -1))
        v[:, : m.vdim, : m.kv_rank].copy_(uv.view(m.heads, m.vdim, -1))

    def _kv_maps(self, i: int) -> Tuple[torch.Tensor, torch.Tensor]:
        """Key maps ``[heads, dim_p, rank_p]`` and value maps ``[heads, vdim_p, rank_p]``."""
        m, w = self.cfg.layers[i].mixer, self.p[f"l{i}.w_ukv"]
        n = m.heads * m.dim_p
        return w[:n].view(m.heads, m.dim_p, -1), w[n:].view(m.heads, m.vdim_p, -1)

    def put_o(self, i: int, wo: torch.Tensor) -> None:
        m, d = self.cfg.layers[i].mixer, self.cfg.width
        self.p[f"l{i}.wo"].view(-1, m.heads, m.vdim_p)[:d, :, : m.vdim].copy_(wo.view(d, m.heads, m.vdim))

    def put_dense(self, i: int, up: torch.Tensor, down: torch.Tensor) -> None:
        d, f = self.cfg.width, self.cfg.layers[i].mlp.ff
        self._ff_rows(i)[:f, :d].copy_(up)
        self.p[f"l{i}.w_down"][:d, :f].copy_(down)

    def put_router(self, i: int, w: torch.Tensor) -> None:
        self._ff_rows(i)[: w.shape[0], : self.cfg.width].copy_(w)

    def _ff_rows(self, i: int) -> torch.Tensor:
        """The feed-forward's rows of the input projection."""
        m = self.cfg.layers[i].mixer
        return self.p[f"l{i}.w_in"][m.q_in + m.kv_in:]

    def put_expert(self, i: int, s: int, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> None:
        d, e = self.cfg.width, self.cfg.layers[i].mlp
        both = self.p[f"l{i}.w_gate_up"][s]
        both[: e.ff, :d].copy_(gate)
        both[e.ff_p:e.ff_p + e.ff, :d].copy_(up)
        self.p[f"l{i}.w_down"][s, :d, : e.ff].copy_(down)

    # ------------------------------------------------------------------ what the generator asks
    def rotations(self) -> Iterable[Tuple[float, int]]:
        return [(l.mixer.rot_base, l.mixer.rot_dim) for l in self.cfg.layers]

    def head_weight(self) -> torch.Tensor:
        return self.p["head"]

    def lasting_caches(self) -> set:
        return {l.mixer.kv_from for l in self.cfg.layers if l.mixer.kv_from is not None}

    def first_visible_key(self, pos: int) -> int:
        """Smallest position any layer still reads once every later token stands at ``pos`` or beyond."""
        return min((max(0, pos - l.mixer.window + 1) if l.mixer.window else 0) for l in self.cfg.layers)

    # ------------------------------------------------------------------ forward
    def _forms_keys(self, m: LatentMixer, spans: _Spans) -> bool:
        """Whether a prefill forms the keys and values it sees (cost: every visible row through the maps, then narrow products per pair) or
        scores the latents (cost: every query through the maps, then wide products per pair, in tiles of up to 32 heads)."""
        if self.f32 or not K.latent_prefill_fits(m.dim_p, m.rot_p, m.vdim_p) or m.scale <= 0:
            return False
        maps = m.heads * m.kv_rank * (m.dim + m.vdim)
        pairs = spans.pairs(m.window)
        formed = maps * spans.total(m.window) + pairs * m.heads * (m.dim + m.rot_dim + 2 * m.vdim)
        scored = maps * sum(spans.lens) + pairs * -(-m.heads // 32) * 128 * 2 * m.row_width
        return formed <= scored

    def _attention(self, i: int, h: torch.Tensor, proj, pos, slot, page_table, cache, decode: bool, form, attend, ff=None) -> torch.Tensor:
        """Attention of layer ``i`` up to the output projection's operand ``[T, heads * vdim_p]``; ``cache`` is the cache it reads (and, if it is
        the layer's own, appends to). ``form``: keys and values are formed (a prefill's spans), else ``attend(m, q)`` scores the latents.
        ``ff``: (column of ``proj``, buffer) of a dense feed-forward whose activation is taken along."""
        m, p, T, eps = self.cfg.layers[i].mixer, self.p, h.shape[0], self.cfg.norm_eps
        bf = dict(dtype=self.dtype, device=self.device)
        cos_t, sin_t = self._tables.get((m.rot_base, m.rot_dim), (None, None))
        kv = (m.q_in, m.kv_rank, p[f"l{i}.kv_norm"], cache, page_table) if m.kv_from is None else None
        src = proj
        if m.q_rank:
            cq = torch.empty((T, m.q_rank_p), **bf)
            K.latent_rows(proj, pos, slot, cos_t, sin_t, m.rot_dim, m.rot_p, eps, q_latent=(0, m.q_rank, p[f"l{i}.q_norm"], cq), kv=kv, ff=ff)
            src, kv, ff = self._lin(cq, p[f"l{i}.w_uq"], decode, ws=1), None, None
        if isinstance(src, K.Partials):
            q = None
            nope = torch.empty((T, m.heads * m.dim_p), **bf)
        else:
            q = src[:, : m.q_width].unflatten(1, (m.heads, m.head_width))
            nope = None
        wide = None if form else torch.empty((T, m.heads, m.row_width), **bf)
        rotated = q[:, :, m.dim_p:] if form else wide[:, :, m.rank_p:]
        K.latent_rows(src, pos, slot, cos_t, sin_t, m.rot_dim, m.rot_p, eps, kv=kv, queries=(0, m.heads, m.dim_p, nope, rotated), ff=ff)
        uk, uv = self._kv_maps(i)
        if form:
            return form(i, m, q)
        K.head_gemm(q[:, :, : m.dim_p] if nope is None else nope.view(T, m.heads, m.dim_p), uk, wide[:, :, : m.rank_p], transposed=True)
        avg = attend(i, m, wide)
        out = torch.empty((T, m.heads, m.vdim_p), **bf)
        return K.head_gemm(avg, uv, out).view(T, -1)

    def _feed_forward(self, i: int, h: torch.Tensor, first, counts: torch.Tensor, decode: bool):
        """What the feed-forward adds to the stream, as a source of ``stream_update``. ``first``: a mixture's router logits, or a dense one's
        activation (None: not computed yet)."""
        p, e = self.p, self.cfg.layers[i].mlp
        if e is None:
            return None
        if isinstance(e, DenseFF):
            act = K.ff_first(h, self._ff_rows(i), "relu2") if first is None else first
            return self._lin(act, p[f"l{i}.w_down"], decode, ws=1)
        ids, wts, ticket = K.moe_route(first, e.experts, e.top, counts, sigmoid=True)
        r = K.moe_dispatch(h, ids, wts, ticket, counts, e.experts, weigh_inputs=True)
        act = K.moe_gemm(r.x_sorted, p[f"l{i}.w_gate_up"], r, e.experts, 0, act="swiglu")
        return K.MoEOutput(K.moe_gemm(act, p[f"l{i}.w_down"], r, e.experts, 0), r.row_of, r.weights, 0)

    def _run(self, tokens, pos, slot, page_table, kcache, decode: bool, form, attend, trace=None) -> torch.Tensor:
        """All layers on ``T`` tokens. ``form(layer)`` gives the way of a layer's attention. Returns the hidden rows the logits are taken from,
        ``[T, width_p]``."""
        cfg, p = self.cfg, self.p
        T = tokens.numel()
        x = torch.empty((T, cfg.width_p), dtype=torch.float32, device=self.device)
        counts = torch.zeros((cfg.n_layers, self.max_experts), dtype=torch.int32, device=self.device)

        def update(a, b, i: int, **kw) -> torch.Tensor:
            name = "final_norm" if i == cfg.n_layers else f"l{i}.norm1"
            return K.stream_update(a, b, self.alpha[i], p[name], p[name + ".b"], x, **kw)

        h = update(p["embed"], None, 0, ids=tokens)
        for i, layer in enumerate(cfg.layers):
            m, e = layer.mixer, layer.mlp
            w_in, n_attn = p[f"l{i}.w_in"], m.q_in + m.kv_in
            first, ff_act = None, None
            if decode or self.f32:                                  # fp32 results: the feed-forward's rows ride along
                proj = self._lin(h, w_in, decode)
                if isinstance(e, DenseFF):
                    first = torch.empty((T, e.ff_p), dtype=self.dtype, device=self.device)
                    ff_act = (n_attn, first)
                elif e is not None:
                    first = proj[:, n_attn:] if self.f32 else proj.columns(n_attn)
            else:
                proj = self._lin(h, w_in[:n_attn], False)
                if isinstance(e, InputScaledMixture):
                    first = self._lin(h, w_in[n_attn:], False, f32_out=True)
            own = i if m.kv_from is None else m.kv_from
            o = self._attention(i, h, proj, pos, slot, page_table, kcache[own], decode, form(i, m) if form else None, attend, ff_act)
            ff = self._feed_forward(i, h, first, counts[i], decode)
            o = self._lin(o, p[f"l{i}.wo"], decode)
            h = update(o, ff, i + 1)
            if trace is not None:
                trace.append(x[:, : cfg.width].clone())
        return h

    def prefill(self, tokens, pos, cu, max_len: int, slot, page_table, kcache, vcache, trace=None, spans=None) -> torch.Tensor:
        """Packed portions of prompts: request ``b`` owns tokens ``cu[b] .. cu[b + 1]`` at consecutive positions ``pos`` (whatever
        came before them is in the cache already), ``slot`` names every token's page-table row; ``spans``: (starts, lengths) of the
        portions on the host. Returns hidden rows ``[T, width_p]``."""
        seen = _Spans(*spans, self.device)

        def formed(i: int, m: LatentMixer, q: torch.Tensor) -> torch.Tensor:
            total, off, lo = seen.rows(m.window)
            rows = K.latent_gather(kcache[i if m.kv_from is None else m.kv_from], page_table, slot, cu, off, lo, total)
            kv = K.gemm(rows[:, : m.rank_p], self.p[f"l{i}.w_ukv"])
            return K.latent_prefill(q, kv, rows, m.dim_p, m.vdim_p, m.rank_p, cu, pos, off, lo, max_len, window=m.window, scale=m.scale,
                                    sink=self.sink[i])

        def attend(i: int, m: LatentMixer, q: torch.Tensor) -> torch.Tensor:
            return self._score_latents(i, m, q, kcache, page_table, slot, pos, None, 1, None)

        return self._run(tokens, pos, slot, page_table, kcache, False, lambda i, m: formed if self._forms_keys(m, seen) else None, attend, trace)

    def _score_latents(self, i: int, m: LatentMixer, q, kcache, page_table, slot, pos, lens, nsplit: int, scratch) -> torch.Tensor:
        cache = kcache[i if m.kv_from is None else m.kv_from]
        kw = dict(window=m.window, scale=m.scale, lens=lens, sink=self.sink[i])
        if not self.f32 and m.scale > 0 and K.latent_decode_fits(m.rank_p, m.row_width):
            return K.latent_decode(q, cache, m.rank_p, page_table, slot, pos, nsplit=nsplit, scratch=scratch, **kw)
        return K.latent_attn_rows(q, cache, m.rank_p, page_table, slot, pos, **kw)

    def _nsplit(self, m: LatentMixer, rows: int, table_pages: int) -> int:
        """Splits of a decode row's pages: the fewest page times over all waves of CTAs, where a CTA costs about four pages on
        top of its own (pipeline fill, merge). One where the CUDA cores score the latents."""
        per_sm = K.latent_decode_ctas_per_sm(m.rank_p, m.row_width)
        if per_sm == 0:
            return 1
        pages = min(table_pages, (m.window - 2) // K.KV_PAGE + 2) if m.window else table_pages
        ctas, slots = rows * -(-m.heads // 32), self._num_sms * per_sm
        return min(range(1, min(pages, 16) + 1), key=lambda n: (-(-ctas * n // slots) * (-(-pages // n) + 4), n))

    def _split_buffer(self, rows: int, table_pages: int) -> torch.Tensor:
        """Scratch of the split attention for ``rows`` rows; kept for good, captured graphs point into it."""
        key = (rows, table_pages)
        if key not in self._split:
            mixers = [l.mixer for l in self.cfg.layers]
            need = max(K.latent_decode_scratch(rows, m.heads, m.rank_p, self._nsplit(m, rows, table_pages)) for m in mixers)
            self._split[key] = torch.empty(max(need, 1), dtype=torch.float32, device=self.device)
        return self._split[key]

    def decode_step(self, token, pos, slot_ids, seq_len, page_table, kcache, vcache, nsplit: int = 1, groups=None) -> torch.Tensor:
        """One token per row (``seq_len = pos + 1`` visible keys, 0 for a retired row). Returns hidden rows ``[B, width_p]``."""
        B, table_pages = token.shape[0], page_table.shape[1]
        scratch = None if self.f32 else self._split_buffer(B, table_pages)

        def attend(i: int, m: LatentMixer, q: torch.Tensor) -> torch.Tensor:
            return self._score_latents(i, m, q, kcache, page_table, slot_ids, pos, seq_len, self._nsplit(m, B, table_pages), scratch)

        return self._run(token, pos, slot_ids, page_table, kcache, True, None, attend)
