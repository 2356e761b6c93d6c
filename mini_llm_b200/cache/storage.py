"""Device memory of the caches, and the view of it each run entry gets.

Per paged group: keys and values as ``[entries, n_pages, page_size, kv_heads,
head_size]`` each (one page id covers every entry of the group, and every
entry's pages are one contiguous array), plus the device copy of the block
tables of the step's items, ``[max_items, max_blocks]`` int32, refilled before
each step.  Per fixed-state group: ``[entries, max_requests, *shape]``, zeroed
for a slot when a request opens it.

The reference allocates K and V per sequence and per layer
(engine/src/gpt2_gpu.cu:147-159) and passes the pointers in a control block
(engine/src/gpt2_gpu_batch.cu:18-24); here the pools are allocated once.
"""

from __future__ import annotations

import torch

from ..parts.spec import FixedState, PagedKV

_STATE_DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16, "int32": torch.int32}


class LayerCache:
    """What one run entry's mixer may touch."""

    kind = "none"
    writes = False
    group = None


class PagedLayerCache(LayerCache):
    kind = "paged"

    def __init__(self, group, k_pages, v_pages, block_table, page_size, writes):
        self.group = group
        self.k_pages, self.v_pages = k_pages, v_pages      # [n_pages, page_size, kv_heads, head_size]
        self.block_table = block_table                     # [max_items, max_blocks] int32, rows = the step's items
        self.page_size = page_size
        self.writes = writes


class StateLayerCache(LayerCache):
    kind = "state"

    def __init__(self, group, state, writes):
        self.group = group
        self.state = state                                 # [max_requests, *shape], indexed by slot
        self.writes = writes


class CompositeLayerCache(LayerCache):
    """The caches of a run entry whose layer has several parts that keep something."""

    kind = "composite"

    def __init__(self, by_role: dict):
        self.by_role = by_role
        self.writes = all(view.writes for view in by_role.values())

    def of(self, role: str):
        return self.by_role.get(role) or LayerCache()

    def sub(self, prefix: str):
        """The caches whose role starts with ``prefix.``, under the rest of their names: what a part
        that is itself put together from parts hands on to each of them."""
        head = prefix + "."
        return CompositeLayerCache({role[len(head):]: view for role, view in self.by_role.items() if role.startswith(head)})


class CacheStorage:
    def __init__(self, manager, order, dtype: torch.dtype, device, max_items: int, poison: float | None = None):
        """``poison``: a debugging value.  Every page slot holds it until a token is stored
        there, and a page holds it again from the moment it is given back: a kernel that
        reads a slot past a request's length, or through a stale block-table row, then
        reads ``poison`` instead of another request's plausible keys."""
        self.manager = manager
        self.device = device
        self.max_items = int(max_items)
        self.poison = poison
        self.spare_page = True                # every pool has a page past its last (index n_pages)
        self.keys, self.values, self.states, self.block_tables = {}, {}, {}, {}
        for group in manager.groups:
            n_entries = len(group.entries)
            if isinstance(group.need, PagedKV):
                # one page beyond the pool's last: no request ever owns it; steps that are filled up
                # to a round shape let their filler tokens store there
                shape = (n_entries, group.pool.n_pages + 1, manager.page_size, group.need.n_kv_heads,
                         group.need.head_size)
                fill = 0.0 if poison is None else poison
                self.keys[group.index] = torch.full(shape, fill, dtype=dtype, device=device)
                if group.need.has_values:
                    shape = (*shape[:4], group.need.value_size or group.need.head_size)
                    self.values[group.index] = torch.full(shape, fill, dtype=dtype, device=device)
                self.block_tables[group.index] = torch.zeros((self.max_items, group.max_blocks), dtype=torch.int32,
                                                             device=device)
            elif isinstance(group.need, FixedState):
                # one slot beyond the last request's: steps that are filled up to a round shape
                # let their filler tokens keep their state there
                shape = (n_entries, manager.max_requests + 1, *group.need.shape)
                self.states[group.index] = torch.zeros(shape, dtype=_STATE_DTYPES[group.need.dtype], device=device)
        def view_of(key, writes):
            g, position = manager.entry_group[key]
            if manager.groups[g].paged:
                values = self.values[g][position] if g in self.values else None
                return PagedLayerCache(g, self.keys[g][position], values, self.block_tables[g], manager.page_size, writes)
            return StateLayerCache(g, self.states[g][position], writes)

        self.views = []
        for index, entry in enumerate(order):
            owner = index if entry.cache_of is None else entry.cache_of
            writes = entry.cache_of is None
            roles = [key[1] for key in manager.entry_group if isinstance(key, tuple) and key[0] == owner]
            # An entry that reads another's cache may still keep state of a fixed size of its own (a
            # filter's last inputs): those views are its own and written; the owner's paged ones are read.
            own = {}
            if not writes:
                own = {key[1]: view_of(key, True) for key in manager.entry_group if isinstance(key, tuple) and key[0] == index}
                if index in manager.entry_group:
                    own[None] = view_of(index, True)
            if owner in manager.entry_group and own:
                raise ValueError(f"run entry {index} keeps state of its own and reads the cache of entry {owner}, whose one cache "
                                 f"has no name: the owner's part must name what it keeps (cache_need() -> {{name: need}})")
            if owner in manager.entry_group:
                self.views.append(view_of(owner, writes))
            elif roles or own:
                by_role = {role: view_of((owner, role), writes) for role in roles
                           if writes or manager.groups[manager.entry_group[(owner, role)][0]].paged}
                by_role.update({role: view for role, view in own.items() if role is not None})
                self.views.append(CompositeLayerCache(by_role))
            else:
                self.views.append(LayerCache())

        # owners behind the run entries (an embedding that keeps something per request)
        for index in range(len(order), manager.n_owners):
            self.views.append(view_of(index, True) if index in manager.entry_group else LayerCache())

        if poison is not None:
            manager.on_free = self.poison_pages

    def paged_views(self):
        """Every paged view, also those inside the caches of entries with several."""
        for view in self.views:
            for one in (view.by_role.values() if view.kind == "composite" else (view,)):
                if one.kind == "paged":
                    yield one

    def poison_pages(self, group_index: int, pages) -> None:
        """Overwrite pages that went back to their pool (debugging engines only)."""
        index = torch.tensor(list(pages), dtype=torch.int64, device=self.device)
        for store in (self.keys, self.values):
            if group_index in store:
                store[group_index].index_fill_(1, index, self.poison)

    def read_tokens(self, view_index: int, slot: int, first: int, count: int):
        """Keys and values of tokens ``first .. first + count - 1`` of the request in ``slot``
        as run entry ``view_index`` holds them: two tensors [count, kv_heads, head_size],
        gathered through the block table (the reference's test hook copies a layer's rows
        out of its contiguous cache, engine/src/gpt2_gpu.cu:185-195)."""
        view = self.views[view_index]
        if view.kind == "composite":
            view = next((v for v in view.by_role.values() if v.kind == "paged"), view)
        if view.kind != "paged":
            raise ValueError(f"run entry {view_index} keeps no paged keys and values")
        page_size = self.manager.page_size
        row = self.manager.block_table_row(view.group, slot)
        positions = torch.arange(first, first + count, dtype=torch.int64)
        pages = torch.from_numpy(row.astype("int64"))[positions // page_size]
        if count and int(pages.min()) < 0:
            raise ValueError(f"slot {slot} holds no page for some of tokens {first}..{first + count - 1}")
        pages, within = pages.to(self.device), (positions % page_size).to(self.device)
        return (view.k_pages[pages, within].clone(),
                view.v_pages[pages, within].clone() if view.v_pages is not None else None)

    def reset_slot(self, slot: int) -> None:
        """Fixed-size state starts at zero for a new request."""
        for state in self.states.values():
            state[:, slot].zero_()

    def bytes(self) -> int:
        total = 0
        for store in (self.keys, self.values, self.states):
            total += sum(t.numel() * t.element_size() for t in store.values())
        return total
