"""What the served decoder families share: flat weights in bf16 or true fp32, rotary tables, projections, logits, and whole
sequences without a generator.

A family derives from ``ServedDecoder``, lays out its matrices (``FlatLayout``, padded with ``pad8``) and provides

  * ``init_weights(seed)``, ``head_weight()``, ``rotations()`` (every (base, dimensions) its layers rotate with);
  * ``prefill`` and ``decode_step`` over the generator's paged cache, which a call appends to before it attends, so a whole prompt, a
    portion of one and a decoded token give the same hidden rows;
  * ``first_visible_key`` if old keys leave its layers' sight (the generator then gives their pages back).

Matrix rows and columns are padded to multiples of 8 elements with zeros (16-byte rows for TMA), so any size loads.
"""
from __future__ import annotations

from typing import Dict, Iterable, List, Tuple

import torch

from ..ops import kernels as K
from .llama import FlatLayout


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class ServedDecoder:
    """Weights and kernels of one model on one GPU, with the interface the generator drives."""

    cached_prefill = True               # prompts may be fed in portions: attention reads the paged cache
    needs_finite_cache = True           # tensor-core tiles cover whole pages: stale entries must be finite numbers
    prefill_spans = False               # ``prefill`` wants every request's (start, length) on the host as well
    KERNEL_SOURCES: Tuple[str, ...] = ()

    def __init__(self, cfg, layout: FlatLayout, device, *, dtype: torch.dtype, trainable: bool):
        if trainable:
            raise ValueError(f"the {cfg.family} family has no backward pass: it is served, not trained")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype} is not supported (bfloat16 or float32)")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        self.f32 = dtype == torch.float32
        self.layout = layout
        self.w = torch.zeros(layout.total, dtype=dtype, device=self.device)
        self.p: Dict[str, torch.Tensor] = {n: layout.view(self.w, n) for n in layout.entries}
        self._ws: Dict[int, torch.Tensor] = {}
        self._tables: Dict[Tuple[float, int], Tuple[torch.Tensor, torch.Tensor]] = {}
        self._outgrown: List[dict] = []      # tables that captured graphs may still read
        self.positions = 0
        self.reserve_positions(cfg.max_pos)
        self._num_sms = torch.cuda.get_device_properties(self.device).multi_processor_count if self.device.type == "cuda" else 148

    # ------------------------------------------------------------------ a family provides
    def rotations(self) -> Iterable[Tuple[float, int]]:
        raise NotImplementedError

    def head_weight(self) -> torch.Tensor:
        raise NotImplementedError

    # ------------------------------------------------------------------ what the generator asks
    def kv_geometry(self) -> List[Tuple[int, int, int]]:
        return self.cfg.kv_geometry()

    def reserve_positions(self, n: int) -> None:
        """Make the rotary tables cover positions below ``n`` (a generator reserves its longest row when it is built)."""
        if n <= self.positions:
            return
        self.positions = n
        self._outgrown.append(self._tables)
        self._tables = {}
        for base, dims in self.rotations():
            if dims and (base, dims) not in self._tables:
                self._tables[(base, dims)] = K.rope_tables(n, dims, base, self.device)

    # ------------------------------------------------------------------ projections
    def _workspace(self, which: int = 0) -> torch.Tensor:
        """Split-K scratch; partials that are alive at the same time take different ones."""
        if which not in self._ws:
            self._ws[which] = torch.empty(32 * 1024 * 1024, dtype=torch.float32, device=self.device)
        return self._ws[which]

    def _lin(self, x: torch.Tensor, w: torch.Tensor, decode: bool, f32_out: bool = False, ws: int = 0):
        """A projection: split-K partials for few rows (the consumer sums them), a plain GEMM otherwise."""
        if self.f32:
            return K.gemm_f32(x, w)
        if decode:
            return K.gemm_partials(x, w, self._workspace(ws))
        return K.gemm(x, w, out_dtype=torch.float32 if f32_out else torch.bfloat16)

    # ------------------------------------------------------------------ whole sequences
    def forward(self, tokens, pos, cu_seqlens, max_seqlen: int, keep: bool = False, kv_sink=None, h_in=None, trace=None):
        """Packed whole sequences without a generator's cache: the keys go to scratch pages, which layers share unless a later layer
        reads an earlier one's. ``trace`` (a list) receives the residual stream after every layer."""
        if keep or kv_sink is not None or h_in is not None:
            raise ValueError(f"the {self.cfg.family} family runs whole sequences for inference only")
        lens = [int(v) for v in (cu_seqlens[1:] - cu_seqlens[:-1]).tolist()]
        self.reserve_positions(max(lens))
        pages = [-(-l // K.KV_PAGE) for l in lens]
        table = torch.zeros((len(lens), max(pages)), dtype=torch.int32)
        first = 1
        for b, n in enumerate(pages):
            table[b, :n] = torch.arange(first, first + n, dtype=torch.int32)
            first += n
        slot = torch.repeat_interleave(torch.arange(len(lens), dtype=torch.int32), torch.tensor(lens)).to(self.device)
        kc, vc = self._scratch_cache(first)
        kw = {"spans": ([0] * len(lens), lens)} if self.prefill_spans else {}
        return self.prefill(tokens, pos, cu_seqlens, max(lens), slot, table.to(self.device), kc, vc, trace=trace, **kw), None

    def _scratch_cache(self, pages: int) -> Tuple[List[torch.Tensor], List[torch.Tensor]]:
        """Pages for one forward pass; layers that keep their keys only while they run lie over one another."""
        geom, lasting = self.kv_geometry(), self.lasting_caches()
        store = {}

        def carve(layer: int, side: int, h: int, width: int) -> torch.Tensor:
            n = pages * h * K.KV_PAGE * width
            key = (side, layer if layer in lasting else -1)
            if key not in store:
                biggest = n if layer in lasting else max(pages * g[0] * K.KV_PAGE * g[1 + side] for g in geom)
                store[key] = torch.zeros(biggest, dtype=self.dtype, device=self.device)
            return store[key][:n].view(pages, h, K.KV_PAGE, width)

        return [carve(i, 0, g[0], g[1]) for i, g in enumerate(geom)], [carve(i, 1, g[0], g[2]) for i, g in enumerate(geom)]

    def lasting_caches(self) -> set:
        """Layers whose cache a later layer reads."""
        return set()

    # ------------------------------------------------------------------ heads
    def lm_logits(self, xf: torch.Tensor, decode: bool = False) -> torch.Tensor:
        """Logits ``[rows, vocab]`` (bf16, or fp32 in an fp32 model)."""
        w = self.head_weight()
        if self.f32:
            return K.gemm_f32(xf, w)[:, : self.cfg.vocab]
        return K.gemm(xf, w, workspace=self._workspace() if decode else None)[:, : self.cfg.vocab]

    def token_logprobs(self, xf_rows: torch.Tensor, targets: torch.Tensor, chunk: int = 8192, temperature: float = 1.0) -> torch.Tensor:
        """``log p(target)`` of the given hidden rows, at most ``chunk`` rows of logits at a time."""
        out = torch.empty(xf_rows.shape[0], dtype=torch.float32, device=self.device)
        for s in range(0, xf_rows.shape[0], chunk):
            t = targets[s:s + chunk].contiguous()
            _, out[s:s + chunk] = K.sample(self.lm_logits(xf_rows[s:s + chunk]), temperature, True, 0, forced=t)
        return out
