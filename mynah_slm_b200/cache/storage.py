"""Device storage of the cache, built from a model's cache plan.

Per storage group: the keys of every entry of the group, each [n_pages,
kv_heads, 64, head_dim] in the run's type, in one allocation, and the values
likewise with their own width and, where several key heads share a value
head, their own number of heads (a group whose mixers keep one vector per
position has none). Beside them: the fixed-size per-sequence state of the
entries (and of the embedding) that ask for one, [max_seqs + 1, *shape]: a sequence's row is zeroed
whenever its slot is handed out; the last row belongs to no sequence and is
there for a step's padding rows.

The page bookkeeping itself is on the host (`SequencePages`).
"""
from __future__ import annotations

from typing import Optional

import torch

from ..parts.base import CacheView
from .pages import PAGE_TOKENS, CacheError, SequencePages


class Cache:
    def __init__(self, plan, n_pages: int, max_seqs: int, dtype: torch.dtype, device):
        self.plan = plan
        self.n_pages, self.max_seqs = n_pages, max_seqs
        self.pages = SequencePages(plan.groups, n_pages, max_seqs)
        self.keys: list[torch.Tensor] = []
        self.values: list[Optional[torch.Tensor]] = []
        for g in plan.groups:
            n = max(len(g.entries), 1)
            vd = g.head_dim if g.v_head_dim is None else g.v_head_dim
            self.keys.append(torch.empty((n, n_pages, g.kv_heads, PAGE_TOKENS, g.head_dim), dtype=dtype, device=device))
            vh = g.kv_heads if getattr(g, "v_heads", None) is None else g.v_heads
            self.values.append(torch.empty((n, n_pages, vh, PAGE_TOKENS, vd), dtype=dtype, device=device) if vd else None)
        self._state_tensors: list[torch.Tensor] = []

        def make(req):
            # one tensor a request, a dictionary of tensors for a mapping of requests
            if req is None:
                return None
            if isinstance(req, dict):
                return {name: make(r) for name, r in req.items()}
            t = torch.zeros((max_seqs + 1, *req.shape), dtype=req.dtype, device=device)
            self._state_tensors.append(t)
            return t

        self.states: dict[int, object] = {}
        self.block_states: dict[int, object] = {}
        for i, e in enumerate(plan.entries):
            if e.state is not None:
                self.states[i] = make(e.state)
            if getattr(e, "block_state", None) is not None:
                self.block_states[i] = make(e.block_state)
        self.embedding_state = make(getattr(plan, "embedding_state", None))
        self.views: list[CacheView] = []
        for i, e in enumerate(plan.entries):
            src = plan.entries[e.source] if e.source is not None else e
            k = v = None
            if src.group is not None:
                k = self.keys[src.group][src.index_in_group]
                v = self.values[src.group][src.index_in_group] if self.values[src.group] is not None else None
            self.views.append(CacheView(group=src.group if src.group is not None else 0, k=k, v=v,
                                        writes=e.source is None, state=self.states.get(i),
                                        block_state=self.block_states.get(i)))

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in [*self.keys, *self.values, *self._state_tensors] if t is not None)

    def open(self) -> int:
        slot = self.pages.open()
        for t in self._state_tensors:
            t[slot].zero_()
        return slot

    def close(self, slot: int) -> None:
        self.pages.close(slot)
