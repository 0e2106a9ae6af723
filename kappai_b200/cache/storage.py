"""Device memory of the cache: page pools and state slots.

For a page group with ``L`` caches (one per schedule entry that keeps keys and
values in it) the pool is one tensor ``[L, n_pages, 2, G, page_size, hd]`` (1 in
the place of 2 where an entry is one row) in the compute dtype: page ``p`` exists in all ``L`` layers at once, so one block
table serves the whole group (the reference keeps ``[layer][kv head][pos][hd]``
per session, src/backend/cpu/common.c:1494-1601).  State of fixed size is one
tensor ``[n_slots, *shape]`` per schedule entry that keeps one.  An entry whose
mixer keeps several memories has one view for each, in a :class:`CompositeView`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Hashable, List, Optional, Tuple, Union

import torch

from .spec import CompositeSpec, PagedKVSpec, StateSpec, leaf_specs


@dataclass
class KVLayerView:
    """One schedule entry's keys and values: ``tensor`` is
    [n_pages, planes, G, page_size, hd]; ``writes`` is False for an entry that only
    reads another entry's cache."""

    group: Hashable
    tensor: torch.Tensor
    writes: bool = True


@dataclass
class StateView:
    tensor: torch.Tensor           # [n_slots, *shape]
    writes: bool = True


@dataclass
class CompositeView:
    parts: Tuple[object, ...]      # the views of a CompositeSpec's parts, in its order


class CacheStorage:
    def __init__(self, specs: List[Optional[object]], cache_of: List[Optional[int]], n_pages: Dict[Hashable, int],
                 page_size: int, n_slots: int, dtype: torch.dtype, device: torch.device):
        """``specs[i]`` is what schedule entry ``i`` asks for (None for an entry
        without a cache, or for one that borrows: ``cache_of[i]`` then names the
        lender).  ``n_pages`` gives the pool size of each page group."""
        self.page_size, self.n_slots = page_size, n_slots
        self.groups: Dict[Hashable, PagedKVSpec] = {}
        members: Dict[Hashable, int] = {}                              # group -> caches in it
        for i, s in enumerate(specs):
            for leaf in leaf_specs(s) if cache_of[i] is None else ():
                if isinstance(leaf, PagedKVSpec):
                    self.groups.setdefault(leaf.group_key, leaf)
                    members[leaf.group_key] = members.get(leaf.group_key, 0) + 1
        self.pools: Dict[Hashable, torch.Tensor] = {}
        for gk, n_caches in members.items():
            s = self.groups[gk]
            self.pools[gk] = torch.zeros((n_caches, n_pages[gk], s.planes, s.num_kv_heads, page_size, s.head_dim),
                                         dtype=dtype, device=device)
        taken = {gk: 0 for gk in members}

        def view_of(s):
            if isinstance(s, CompositeSpec):
                return CompositeView(tuple(view_of(p) for p in s.parts))
            if isinstance(s, PagedKVSpec):
                gk = s.group_key
                taken[gk] += 1
                return KVLayerView(gk, self.pools[gk][taken[gk] - 1], True)
            if isinstance(s, StateSpec):
                dt = getattr(torch, s.dtype)
                return StateView(torch.zeros((n_slots,) + tuple(s.shape), dtype=dt, device=device), True)
            return None

        self.views: List[Optional[object]] = [view_of(s) if cache_of[i] is None else None for i, s in enumerate(specs)]
        for i, src in enumerate(cache_of):
            if src is not None:
                v = self.views[src]
                if v is None:
                    raise ValueError(f"schedule entry {i} borrows the cache of entry {src}, which keeps none")
                self.views[i] = _read_only(v)

    def bytes_per_token(self, group: Hashable) -> int:
        """Bytes an entry takes in all caches of the group (a token, where the group keeps one entry a position)."""
        t = self.pools[group]
        return t[:, 0, :, :, 0, :].numel() * t.element_size()

    def total_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in list(self.pools.values()) + self.state_tensors())

    def state_tensors(self) -> List[torch.Tensor]:
        """The tensors of fixed-size state (borrowed ones not counted again)."""
        out: List[torch.Tensor] = []

        def collect(v):
            if isinstance(v, CompositeView):
                for p in v.parts:
                    collect(p)
            elif isinstance(v, StateView) and v.writes:
                out.append(v.tensor)

        for v in self.views:
            collect(v)
        return out


def _read_only(v: Union[KVLayerView, StateView, CompositeView]):
    """A borrower's view of what another entry keeps."""
    if isinstance(v, CompositeView):
        return CompositeView(tuple(_read_only(p) for p in v.parts))
    if isinstance(v, KVLayerView):
        return KVLayerView(v.group, v.tensor, False)
    return StateView(v.tensor, False)
