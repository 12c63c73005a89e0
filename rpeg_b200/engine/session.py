"""Feeding a generator by hand: requests arrive, bring any number of tokens per step, and leave.

``Generator.generate`` owns a whole batch from prompt to last token. A ``Session`` hands the same slots, page pool, prefill
and decode step to a caller who decides what each request feeds next (scoring, replaying a recorded schedule, an outer
server loop). One ``feed`` call is one engine step over any mix of requests: single tokens that continue a request go through
the decode step, everything else through the prefill, each continuing from what the request has in the cache.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import torch

from ..ops import kernels as K
from .generation import PAGE, Generator, PagePool


@dataclass
class _Request:
    slot: int
    length: int = 0                                     # tokens in the cache
    gone: int = 0                                       # leading pages given back (never read again)
    pages: List[int] = field(default_factory=list)


class Session:
    def __init__(self, gen: Generator):
        """Takes over the generator's slots and pages (``generate`` starts afresh afterwards)."""
        self.gen = gen
        gen.pool = PagePool(gen.pool.num_pages)
        gen.page_table.zero_()
        if gen.zero_cache:
            gen.kv_storage.zero_()
        self.requests: Dict[Hashable, _Request] = {}
        self.free_slots = list(range(gen.max_slots - 1, -1, -1))
        self.rows = torch.arange(gen.max_slots, dtype=torch.int32, device=gen.dev)

    # ------------------------------------------------------------------ pages
    def _reserve(self, q: _Request, n: int) -> None:
        """Pages for ``n`` more tokens of the request."""
        have = q.gone + len(q.pages)
        need = -(-(q.length + n) // PAGE) - have
        if need > 0:
            new = self.gen.pool.take(need)
            q.pages.extend(new)
            self.gen.page_table[q.slot, have:have + need] = torch.tensor(new, dtype=torch.int32, device=self.gen.dev)

    def _drop_passed(self, q: _Request) -> None:
        """Give back the pages no later token of the request reads."""
        if self.gen.first_visible_key is None:
            return
        k = min(self.gen.first_visible_key(q.length) // PAGE - q.gone, len(q.pages))
        if k > 0:
            self.gen.pool.give(q.pages[:k])
            del q.pages[:k]
            self.gen.page_table[q.slot, q.gone:q.gone + k] = 0
            q.gone += k

    def end(self, rid: Hashable) -> None:
        """The request is finished: its pages and its slot go back."""
        q = self.requests.pop(rid)
        self.gen.pool.give(q.pages)
        self.gen.page_table[q.slot] = 0
        self.free_slots.append(q.slot)

    # ------------------------------------------------------------------ one step
    def _decode(self, reqs: Sequence[_Request], tokens: Sequence[int]) -> torch.Tensor:
        """Hidden rows of one more token per request, through the decode step on a table of just these requests' rows."""
        g, b = self.gen, len(reqs)
        i32 = dict(dtype=torch.int32, device=g.dev)
        pos = torch.tensor([q.length for q in reqs], **i32)
        table = g.page_table[torch.tensor([q.slot for q in reqs], dtype=torch.long, device=g.dev)]
        return g.model.decode_step(torch.tensor(list(tokens), **i32), pos, self.rows[:b], pos + 1, table, g.kcache, g.vcache, nsplit=g._nsplit(b))

    @torch.no_grad()
    def feed(self, entries: Sequence[Tuple[Hashable, Sequence[int], Sequence[int]]]) -> List[Optional[torch.Tensor]]:
        """``(request, its next tokens, places among them whose logits are wanted)`` per entry; unknown requests start.
        Returns the logits ``[wanted, vocab]`` per entry (None where nothing is wanted)."""
        g = self.gen
        if len({rid for rid, _, _ in entries}) != len(entries):
            raise ValueError("a request may appear once per step")
        for rid, tokens, want in entries:
            if not len(tokens):
                raise ValueError(f"request {rid!r} brings no tokens")
            if min(tokens) < 0 or max(tokens) >= g.cfg.vocab:
                raise ValueError(f"request {rid!r} brings a token outside the vocabulary")
            if len(want) and (min(want) < 0 or max(want) >= len(tokens)):
                raise ValueError(f"request {rid!r} wants a place outside its tokens")
            have = self.requests[rid].length if rid in self.requests else 0
            if have + len(tokens) > g.max_seq_len:
                raise ValueError(f"request {rid!r} of {have + len(tokens)} tokens exceeds max_seq_len ({g.max_seq_len})")
        new = [rid for rid, _, _ in entries if rid not in self.requests]
        if len(new) > len(self.free_slots):
            raise RuntimeError(f"{len(new)} new requests but only {len(self.free_slots)} of {g.max_slots} slots are free")
        for rid in new:
            self.requests[rid] = _Request(self.free_slots.pop())
        reqs = [self.requests[rid] for rid, _, _ in entries]
        for q, (_, tokens, _) in zip(reqs, entries):
            self._reserve(q, len(tokens))
        out: List[Optional[torch.Tensor]] = [None] * len(entries)
        single = [i for i, q in enumerate(reqs) if q.length > 0 and len(entries[i][1]) == 1]
        many = [i for i in range(len(entries)) if i not in set(single)]
        if single:
            hidden = self._decode([reqs[i] for i in single], [entries[i][1][0] for i in single])
            rows = [j for j, i in enumerate(single) if len(entries[i][2])]
            if rows:
                logits = g.model.lm_logits(hidden, decode=True)
                for j in rows:
                    out[single[j]] = logits[j].expand(len(entries[single[j]][2]), -1)
        serial = [i for i in many if reqs[i].length > 0 and not g.cached_prefill]      # no prefill behind a cached prefix
        packed = [i for i in many if i not in set(serial)]
        if packed:
            hidden, cu = g.prefill_hidden([torch.tensor(list(entries[i][1]), dtype=torch.int32) for i in packed], [reqs[i].slot for i in packed],
                                          [reqs[i].length for i in packed])
            offs = cu.tolist()
            rows = [offs[j] + int(w) for j, i in enumerate(packed) for w in entries[i][2]]
            if rows:
                logits = g.model.lm_logits(K.gather_rows(hidden, torch.tensor(rows, dtype=torch.int32, device=g.dev)))
                at = 0
                for i in packed:
                    n = len(entries[i][2])
                    out[i] = logits[at:at + n] if n else None
                    at += n
        for i in serial:
            _, tokens, want = entries[i]
            got = []
            for t in tokens:
                got.append(self._decode([reqs[i]], [t]))
                reqs[i].length += 1
            if len(want):
                out[i] = g.model.lm_logits(torch.cat([got[w] for w in want]), decode=True)
        for i, q in enumerate(reqs):
            if i not in set(serial):
                q.length += len(entries[i][1])
            self._drop_passed(q)
        return out
