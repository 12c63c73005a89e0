"""Dulisun decoder: chunked attention whose values are the projected keys, a softmax sink, norms on the sublayers' outputs
around an fp32 residual stream, and grouped-router mixtures of experts. Every layer has its own sizes.

    x  = norm(E[token])
    x += norm1( W_o attention(x) )             q = W_q x, k = W_k x, v = k; interleaved rotary, then unit RMS per head
    x += norm2( sum_e s_e expert_e(x) + shared(x) )        (layers without a feed-forward skip this)
    logits = E norm(x)

What runs where:
  * the residual stream, norms, rotary angles, scores, softmax and routing are fp32; the matrix products take the bf16
    copy of the stream that the norm kernels write next to it (``dtype=torch.float32`` runs everything in true fp32);
  * one kernel per place the stream is touched (``ops.kernels.residual_norm``): it sums the split-K partials of the
    projection before it, or the weighted expert outputs, normalises, adds to the stream and writes the next operand; the
    norm before the logits rides on the last of them;
  * keys (rotated, normalised) and values (the raw projection) live in the generator's paged cache. A whole prompt, a
    portion of one and a decoded token append to it first and then attend over it, so nothing depends on how a prompt was
    cut. No key before the current chunk is ever read again (``first_visible_key``): the generator gives those pages back;
  * a shared feed-forward wider than the routed experts is stored as several always-on experts of their size (its hidden
    units are independent), so routed and shared experts are one grouped GEMM up and one down.

This family is served (generation, log-probs); it has no backward pass here.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, Iterable, List, Optional, Tuple

import torch

from ..ops import kernels as K
from .llama import FlatLayout
from .served import ServedDecoder, pad8


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int = 0                     # keys are visible inside chunks of this many positions; 0: all earlier keys
    rot_dims: int = 0                   # leading dimensions that are rotated (interleaved pairs)
    rot_base: float = 10000.0

    @property
    def dim_p(self) -> int:
        return pad8(self.dim)

    @property
    def q_width(self) -> int:
        return self.heads * self.dim_p

    @property
    def k_width(self) -> int:
        return self.kv_heads * self.dim_p


@dataclass(frozen=True)
class ExpertMixture:
    experts: int
    top: int
    ff: int
    shared_ff: int = 0                  # hidden size of the always-on feed-forward; 0: none
    groups: int = 1
    keep: int = 1                       # groups a token may choose from

    @property
    def ff_p(self) -> int:
        return pad8(self.ff)

    @property
    def n_shared(self) -> int:
        """Always-on experts of size ``ff`` that hold the shared feed-forward."""
        return -(-self.shared_ff // self.ff)

    @property
    def segments(self) -> int:
        return self.experts + self.n_shared


@dataclass(frozen=True)
class DecoderLayer:
    mixer: AttentionMixer
    mlp: Optional[ExpertMixture] = None


@dataclass(frozen=True)
class DulisunConfig:
    width: int
    vocab: int
    layers: Tuple[DecoderLayer, ...]
    norm_eps: float = 1e-6
    max_pos: int = 4096                 # initial size of the rotary tables (they grow with the generator's row length)
    family: str = "dulisun"

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
        """(KV heads, key width, value width) of every layer's cache."""
        if tp != 1:
            raise ValueError("this family has no tensor-parallel cache layout")
        return [(l.mixer.kv_heads, l.mixer.dim_p, l.mixer.dim_p) for l in self.layers]

    def n_params(self) -> int:
        return DulisunLayout(self).total


class DulisunLayout(FlatLayout):
    """Flat offsets of every matrix (padded shapes)."""

    def __init__(self, cfg: DulisunConfig):
        super().__init__()
        d = cfg.width_p
        self.add("embed", cfg.vocab_p, d)
        self.add("embed_norm", d)
        for i, layer in enumerate(cfg.layers):
            m, e = layer.mixer, layer.mlp
            self.add(f"l{i}.wqk", m.q_width + m.k_width, d)
            self.add(f"l{i}.wo", d, m.q_width)
            self.add(f"l{i}.norm1", d)
            if e is not None:
                self.add(f"l{i}.router", pad8(e.experts), d)
                self.add(f"l{i}.w_up", e.segments, e.ff_p, d)
                self.add(f"l{i}.w_down", e.segments, d, e.ff_p)
                self.add(f"l{i}.norm2", d)
        self.add("final_norm", d)


class DulisunModel(ServedDecoder):
    """Weights and kernels of one model on one GPU."""

    KERNEL_SOURCES = ("gemm.cu", "generate.cu", "loss.cu", "residual_norm.cu", "window_attn.cu", "window_prefill.cu", "moe.cu", "gemm_f32.cu")

    def __init__(self, cfg: DulisunConfig, device, *, dtype: torch.dtype = torch.bfloat16, seed: Optional[int] = 0,
                 trainable: bool = False):
        """``seed=None`` leaves the weights zero (a checkpoint is about to be loaded)."""
        super().__init__(cfg, DulisunLayout(cfg), device, dtype=dtype, trainable=trainable)
        self.sink = [torch.zeros(l.mixer.heads, dtype=torch.float32, device=self.device) for l in cfg.layers]
        self.max_experts = max([l.mlp.experts for l in cfg.layers if l.mlp is not None], default=1)
        self._split: Dict[Tuple[int, int], Tuple[torch.Tensor, torch.Tensor]] = {}
        if seed is not None:
            self.init_weights(seed)

    # ------------------------------------------------------------------ weights
    def init_weights(self, seed: int = 0) -> None:
        """Random weights of the true sizes (the padding stays zero), unit-gain matrices and norms near one."""
        gen = torch.Generator(device=self.device)
        gen.manual_seed(seed)

        def rnd(*shape: int) -> torch.Tensor:
            return torch.randn(shape, generator=gen, device=self.device, dtype=torch.float32)

        d = self.cfg.width
        self.p["embed"][: self.cfg.vocab, :d].copy_(rnd(self.cfg.vocab, d) / math.sqrt(d))
        for name in self.p:
            if name.endswith(("norm", "norm1", "norm2")):
                self.p[name][:d].copy_(0.1 * rnd(d))
        for i, layer in enumerate(self.cfg.layers):
            m, e = layer.mixer, layer.mlp
            self.put_qk(i, rnd(m.heads * m.dim, d) / math.sqrt(d), rnd(m.kv_heads * m.dim, d) / math.sqrt(d))
            self.put_o(i, rnd(d, m.heads * m.dim) / math.sqrt(m.heads * m.dim))
            self.sink[i].copy_(rnd(m.heads))
            if e is not None:
                self.p[f"l{i}.router"][: e.experts, :d].copy_(rnd(e.experts, d) / math.sqrt(d))
                for s in range(e.experts):
                    self.put_expert(i, s, rnd(e.ff, d) / math.sqrt(d), rnd(d, e.ff) / math.sqrt(e.ff))
                if e.shared_ff:
                    self.put_shared(i, rnd(e.shared_ff, d) / math.sqrt(d), rnd(d, e.shared_ff) / math.sqrt(e.shared_ff))

    def put_qk(self, i: int, wq: torch.Tensor, wk: torch.Tensor) -> None:
        """Stack the query and key projections, every head padded to ``dim_p`` rows."""
        m, d = self.cfg.layers[i].mixer, self.cfg.width
        dst = self.p[f"l{i}.wqk"].view(m.heads + m.kv_heads, m.dim_p, -1)
        dst[: m.heads, : m.dim, :d].copy_(wq.view(m.heads, m.dim, d))
        dst[m.heads:, : m.dim, :d].copy_(wk.view(m.kv_heads, m.dim, d))

    def put_o(self, i: int, wo: torch.Tensor) -> None:
        m, d = self.cfg.layers[i].mixer, self.cfg.width
        self.p[f"l{i}.wo"].view(-1, m.heads, m.dim_p)[:d, :, : m.dim].copy_(wo.view(d, m.heads, m.dim))

    def put_expert(self, i: int, s: int, up: torch.Tensor, down: torch.Tensor) -> None:
        """Segment ``s`` of the layer's mixture: up ``[<= ff, width]``, down ``[width, <= ff]``."""
        d, f = self.cfg.width, up.shape[0]
        self.p[f"l{i}.w_up"][s, :f, :d].copy_(up)
        self.p[f"l{i}.w_down"][s, :d, :f].copy_(down)

    def put_shared(self, i: int, up: torch.Tensor, down: torch.Tensor) -> None:
        """The shared feed-forward, cut along its hidden size into always-on experts of size ``ff``."""
        e = self.cfg.layers[i].mlp
        for s in range(e.n_shared):
            self.put_expert(i, e.experts + s, up[s * e.ff:(s + 1) * e.ff], down[:, s * e.ff:(s + 1) * e.ff])

    # ------------------------------------------------------------------ what the generator asks
    def rotations(self) -> Iterable[Tuple[float, int]]:
        return [(l.mixer.rot_base, l.mixer.rot_dims) for l in self.cfg.layers]

    def head_weight(self) -> torch.Tensor:
        return self.p["embed"]

    def first_visible_key(self, pos: int) -> int:
        """Smallest position any layer still reads once every later token stands at ``pos`` or beyond."""
        return min((pos // l.mixer.window * l.mixer.window if l.mixer.window else 0) for l in self.cfg.layers)

    # ------------------------------------------------------------------ forward
    def _mixture(self, i: int, e: ExpertMixture, h: torch.Tensor, counts: torch.Tensor, decode: bool) -> K.MoEOutput:
        p = self.p
        logits = self._lin(h, p[f"l{i}.router"], decode, f32_out=True)
        ids, wts, ticket = K.moe_route(logits, e.experts, e.top, counts, n_groups=e.groups, keep_groups=e.keep)
        r = K.moe_dispatch(h, ids, wts, ticket, counts, e.experts)
        act = K.moe_gemm(r.x_sorted, p[f"l{i}.w_up"], r, e.experts, e.n_shared, shared_x=h if e.n_shared else None, act="gelu")
        y = K.moe_gemm(act, p[f"l{i}.w_down"], r, e.experts, e.n_shared)
        return K.MoEOutput(y, r.row_of, r.weights, e.n_shared)

    def _run(self, tokens, pos, slot, page_table, kcache, vcache, attend, decode: bool, trace=None) -> torch.Tensor:
        """All layers on ``T`` tokens; ``attend(layer, q)`` reads the cache after this call appended to it. Returns the
        hidden rows the logits are taken from, ``[T, width_p]``."""
        cfg, p, d, eps = self.cfg, self.p, self.cfg.width, self.cfg.norm_eps
        T = tokens.numel()
        x = torch.empty((T, cfg.width_p), dtype=torch.float32, device=self.device)
        counts = torch.zeros((cfg.n_layers, self.max_experts), dtype=torch.int32, device=self.device)

        def norm(src, name: str, last: bool, **kw):
            y = K.residual_norm(src, p[name], eps, d, x=x, w2=p["final_norm"] if last else None, want_act=not self.f32, **kw)
            return x if y is None else y

        h = norm(p["embed"], "embed_norm", False, ids=tokens, add=False)
        for i, layer in enumerate(cfg.layers):
            m, e = layer.mixer, layer.mlp
            last = i + 1 == cfg.n_layers
            cos_t, sin_t = self._tables.get((m.rot_base, m.rot_dims), (None, None))
            qk = self._lin(h, p[f"l{i}.wqk"], decode)
            q = torch.empty((T, m.q_width), dtype=self.dtype, device=self.device)
            K.rotary_append(qk, q, 0, m.q_width, m.q_width, slot, pos, cos_t, sin_t, page_table, kcache[i], vcache[i], m.heads, m.dim,
                            m.rot_dims, eps)
            o = self._lin(attend(i, q), p[f"l{i}.wo"], decode)
            h = norm(o, f"l{i}.norm1", last and e is None)
            if e is not None:
                h = norm(self._mixture(i, e, h, counts[i], decode), f"l{i}.norm2", last)
            if trace is not None:
                trace.append(x[:, :d].clone())
        return h

    def prefill(self, tokens, pos, cu, max_len: int, slot, page_table, kcache, vcache, trace=None) -> torch.Tensor:
        """Packed portions of prompts: request ``b`` owns tokens ``cu[b] .. cu[b + 1]`` at consecutive positions ``pos`` (whatever
        came before them is in the cache already), ``slot`` names every token's page-table row. Returns hidden rows ``[T, width_p]``."""
        def attend(i: int, q: torch.Tensor) -> torch.Tensor:
            m = self.cfg.layers[i].mixer
            if not self.f32 and m.dim_p <= K.WINDOW_PREFILL_MAX_DIM and m.scale > 0:
                return K.window_prefill(q, kcache[i], vcache[i], page_table, cu, pos, slot, max_len, m.heads, window=m.window, scale=m.scale,
                                        sink=self.sink[i])
            return K.rows_attn(q, kcache[i], vcache[i], page_table, slot, pos, m.heads, window=m.window, scale=m.scale, sink=self.sink[i])

        return self._run(tokens, pos, slot, page_table, kcache, vcache, attend, False, trace)

    def _nsplit(self, m: AttentionMixer, rows: int, table_pages: int) -> int:
        """Splits of a decode row's pages: the fewest page times over all waves of CTAs, where a CTA costs about four pages on
        top of its own (pipeline fill, merge) and two or three of them share an SM."""
        pages = min(table_pages, m.window // K.KV_PAGE + 2) if m.window else table_pages
        group = m.heads // m.kv_heads
        narrow = (group - 1) % 8 < 4 and group <= 12
        ctas = rows * m.kv_heads * -(-group // (4 if narrow else 8))
        slots = self._num_sms * (3 if narrow else 2)
        return min(range(1, min(pages, 16) + 1), key=lambda n: (-(-ctas * n // slots) * (-(-pages // n) + 4), n))

    def _split_buffers(self, rows: int, table_pages: int) -> Tuple[torch.Tensor, torch.Tensor]:
        """Scratch of the split attention for ``rows`` rows; kept for good, captured graphs point into it."""
        key = (rows, table_pages)
        if key not in self._split:
            mixers = [l.mixer for l in self.cfg.layers]
            need = max(K.rows_attn_scratch(rows, m.heads, m.dim_p, self._nsplit(m, rows, table_pages)) for m in mixers)
            self._split[key] = (torch.empty(max(need, 1), dtype=torch.float32, device=self.device),
                                torch.zeros(rows * max(m.heads for m in mixers), dtype=torch.int32, device=self.device))
        return self._split[key]

    def decode_step(self, token, pos, slot_ids, seq_len, page_table, kcache, vcache, nsplit: int = 1, groups=None) -> torch.Tensor:
        """One token per row (``seq_len = pos + 1`` visible keys, 0 for a retired row). Returns hidden rows ``[B, width_p]``."""
        B, table_pages = token.shape[0], page_table.shape[1]
        scratch, arrive = self._split_buffers(B, table_pages)

        def attend(i: int, q: torch.Tensor) -> torch.Tensor:
            m = self.cfg.layers[i].mixer
            return K.rows_attn(q, kcache[i], vcache[i], page_table, slot_ids, pos, m.heads, window=m.window, scale=m.scale, lens=seq_len,
                               sink=self.sink[i], nsplit=self._nsplit(m, B, table_pages), scratch=scratch, arrive=arrive)

        return self._run(token, pos, slot_ids, page_table, kcache, vcache, attend, True)
