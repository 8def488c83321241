"""Device memory of the cache, laid out for the groups the model's layers form.

`CacheLayout` reads a model's schedule: runs whose mixers keep paged keys/values with the
same (kv heads, head size, window, parts, kept first positions) form a group; each writing run gets a plane of its own in
the group's pool, a run with `cache_of` shares the plane of the run it names (it may look back
over another window: the plane then keeps what the widest of its readers needs).  Runs whose
mixers (or blocks) keep a fixed-size state get a state array [max_requests, ...] indexed by slot
id; a state always belongs to one run, also when the run reads another run's pages, or to the
model's embedding (`embedding_need`), which may look back at a request's tokens.

`CacheStorage` allocates one pool per group, [planes, pages, parts (K, V; or one), kv heads,
page_size, head size] in the compute dtype, the state arrays, and the native `CacheManager` that owns
the page and slot numbers.  Page size and page counts are parameters (the pool is sized for
the tokens the caller wants resident, or for a fraction of the free HBM).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from .. import host


@dataclass
class LayerCache:
    """What one run of a layer may touch."""
    group: Optional[int]            # index into ctx.block_tables, None when the mixer keeps no pages
    plane: Optional[torch.Tensor]   # [pages, 2, Hkv, page_size, D]
    page_stride: int                # elements from one page to the next
    page_size: int
    writes: bool                    # False: reads the plane another run wrote
    state: Optional[torch.Tensor]   # [max_requests, ...] or None


class CacheLayout:
    def __init__(self, model):
        self.needs = model.cache_needs()
        self.schedule = model.schedule
        self.group_keys: List[tuple] = []
        self.group_keep_first: List[int] = []
        self.group_planes: List[int] = []
        self.run_group: List[Optional[int]] = []
        self.run_plane: List[Optional[int]] = []
        self.run_state: List[Optional[int]] = []
        self.state_needs = []
        # the window a writing run's plane must keep: the widest of the runs that read it (0: everything)
        first = {k: need.paged.keep_first for k, (run, need) in enumerate(zip(self.schedule, self.needs))
                 if run.cache_of is None and need.paged is not None}
        keep = {k: [need.paged.window] for k, (run, need) in enumerate(zip(self.schedule, self.needs))
                if run.cache_of is None and need.paged is not None}
        for k, (run, need) in enumerate(zip(self.schedule, self.needs)):
            if run.cache_of is not None:
                j = run.cache_of
                a, b = need.paged, self.needs[j].paged
                if (a is None) != (b is None) or (a is not None and (a.n_kv_heads, a.head_dim, a.parts) !=
                                                  (b.n_kv_heads, b.head_dim, b.parts)):
                    raise ValueError(f"run {k} cannot read the cache of run {j}: their needs differ")
                if a is not None:
                    keep[j].append(a.window)
                    first[j] = max(first[j], a.keep_first)
        for k, (run, need) in enumerate(zip(self.schedule, self.needs)):
            if run.cache_of is not None:
                j = run.cache_of
                self.run_group.append(self.run_group[j])
                self.run_plane.append(self.run_plane[j])
            elif need.paged is not None:
                window = 0 if min(keep[k]) <= 0 else max(keep[k])
                key = (need.paged.n_kv_heads, need.paged.head_dim, window, need.paged.parts)
                kept = first[k] if window else 0
                if (key, kept) not in zip(self.group_keys, self.group_keep_first):
                    self.group_keys.append(key)
                    self.group_keep_first.append(kept)
                    self.group_planes.append(0)
                g = list(zip(self.group_keys, self.group_keep_first)).index((key, kept))
                self.run_group.append(g)
                self.run_plane.append(self.group_planes[g])
                self.group_planes[g] += 1
            else:
                self.run_group.append(None)
                self.run_plane.append(None)
            if need.state is not None:
                self.run_state.append(len(self.state_needs))
                self.state_needs.append(need.state)
            else:
                self.run_state.append(None)

        need = model.embedding_need() if hasattr(model, "embedding_need") else None
        self.embedding_state: Optional[int] = None
        if need is not None and need.state is not None:
            self.embedding_state = len(self.state_needs)
            self.state_needs.append(need.state)

    def bytes_per_token(self, dtype) -> int:
        size = torch.empty((), dtype=dtype).element_size()
        return sum(parts * h * d * planes * size for (h, d, _, parts), planes in zip(self.group_keys, self.group_planes))


class CacheStorage:
    def __init__(self, model, dtype, device, page_size=16, num_pages=None, max_requests=64, max_model_len=None,
                 max_tokens=None):
        """num_pages: pages per group (int or list); or max_tokens: tokens to keep resident,
        from which the page count follows (every group gets enough pages for them)."""
        self.layout = CacheLayout(model)
        self.dtype, self.device, self.page_size = dtype, device, int(page_size)
        n_groups = len(self.layout.group_keys)
        max_model_len = int(max_model_len or 4096)
        if num_pages is None:
            if max_tokens is None:
                raise ValueError("give num_pages or max_tokens")
            num_pages = (int(max_tokens) + self.page_size - 1) // self.page_size
        pages = list(num_pages) if isinstance(num_pages, (list, tuple)) else [int(num_pages)] * n_groups
        self.table_width = (max_model_len + self.page_size - 1) // self.page_size
        specs = [host.module().GroupSpec(self.page_size, key[2], pages[g], self.table_width,
                                         self.layout.group_keep_first[g])
                 for g, key in enumerate(self.layout.group_keys)]
        if not specs:   # a model without paged layers still needs slots and lengths: pages without memory
            specs = [host.module().GroupSpec(self.page_size, 0, int(max_requests) * self.table_width, self.table_width)]
            self._dummy_group = True
        else:
            self._dummy_group = False
        self.manager = host.module().CacheManager(specs, int(max_requests))
        self.max_requests = int(max_requests)
        self.pools = []
        for g, (hkv, d, _w, parts) in enumerate(self.layout.group_keys):
            self.pools.append(torch.empty((self.layout.group_planes[g], pages[g], parts, hkv, self.page_size, d),
                                          dtype=dtype, device=device))
        self.states = [torch.zeros((self.max_requests,) + tuple(n.shape), dtype=n.dtype, device=device)
                       for n in self.layout.state_needs]
        self._views = [self._make_view(k) for k in range(len(self.layout.schedule))]

    def _make_view(self, k):
        lay = self.layout
        g, p, s = lay.run_group[k], lay.run_plane[k], lay.run_state[k]
        plane = self.pools[g][p] if g is not None else None
        stride = plane.stride(0) if plane is not None else 0
        return LayerCache(group=g, plane=plane, page_stride=stride, page_size=self.page_size,
                          writes=lay.schedule[k].cache_of is None, state=self.states[s] if s is not None else None)

    @staticmethod
    def bytes_per_token_of(model, dtype) -> int:
        return CacheLayout(model).bytes_per_token(dtype)

    def layer_cache(self, k) -> LayerCache:
        return self._views[k]

    @property
    def embedding_state(self) -> Optional[torch.Tensor]:
        """The embedding's state rows [max_requests, ...], or None."""
        i = self.layout.embedding_state
        return self.states[i] if i is not None else None

    @property
    def n_groups(self):
        return len(self.pools)

    # ---- requests
    def open(self) -> int:
        slot = self.manager.open()
        for s in self.states:
            s[slot].zero_()          # a new request starts from an all-zero state
        return slot

    def close(self, slot: int) -> None:
        self.manager.close(slot)
