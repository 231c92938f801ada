"""Paged KV pool on the device: 16-token pages, one pool per layer, block tables per sequence.

The pool replaces the reference's per-request growing caches and its block store
(eredu/src/backend/mlx/runtime/cache/kv.rs:2781-2860 chunked growth, :1535-1627 paged truncate):
pages are fixed [n_kv, 16, head_dim] slabs inside two large tensors (K and V) per model shard, so a
sequence's cache is a list of page ids and truncation (speculative rollback) is a length change.
Page 0 is never handed out: padded block-table entries point at it.
"""
from __future__ import annotations

from typing import Optional

import torch

PAGE = 16


class PageAllocator:
    """Free-list page allocator (host side). The C++ block manager (``_eredu_host.BlockManager``) has the
    same interface and is used when the native module is built; this is the portable fallback."""

    def __init__(self, num_pages: int):
        self.num_pages = num_pages
        self._free = list(range(num_pages - 1, 0, -1))

    def free_pages(self) -> int:
        return len(self._free)

    def alloc(self, n: int) -> list[int]:
        if n > len(self._free):
            raise MemoryError(f"KV pool exhausted: need {n} pages, {len(self._free)} free")
        out = self._free[-n:][::-1] if n else []
        del self._free[len(self._free) - n:]
        return out

    def release(self, pages) -> None:
        self._free.extend(reversed(list(pages)))


class PagedKVCache:
    def __init__(self, n_layers: int, n_kv_heads: int, head_dim: int, num_pages: int, dtype, device,
                 first_layer: int = 0, attention_layers=None, conv_layers=None, conv_channels: int = 0, conv_hist: int = 0,
                 value_dim: Optional[int] = None, layer_dims: Optional[dict] = None, donors: Optional[dict] = None,
                 layer_pools: Optional[dict] = None):
        """``layer_dims``: layer -> (kv heads, key width, value width) for families whose layers differ; layers of one
        geometry share a pool tensor, so a page id is valid in every layer. ``donors``: layer -> the earlier layer whose
        keys and values it reads (it keeps none of its own). ``layer_pools``: layer -> tokens of a block whose mean key and
        value are kept as well; a page holds the means of the blocks that end in it, so they come and go with the page.
        ``attention_layers`` / ``conv_layers``: global indices of the layers that keep K/V pages respectively a
        short-convolution state (hybrid models); by default every one of the ``n_layers`` layers keeps K/V.
        The convolution state pool [layer, page, conv_hist, channels] is indexed by a sequence's first page."""
        self.n_kv_heads, self.head_dim = n_kv_heads, head_dim
        self.num_pages = num_pages
        self.first_layer = first_layer
        if attention_layers is None:
            attention_layers = list(range(first_layer, first_layer + n_layers))
        self.n_layers = len(attention_layers)
        default = (n_kv_heads, head_dim, head_dim if value_dim is None else value_dim)
        groups: dict = {}
        for li in attention_layers:
            groups.setdefault(tuple((layer_dims or {}).get(li, default)), []).append(li)
        if not groups:
            groups[default] = []
        self.pools, self._kv_index = [], {}
        for g, ((heads, dk, dv), members) in enumerate(groups.items()):
            k = torch.zeros((len(members), num_pages, heads, PAGE, dk), dtype=dtype, device=device)
            # latent-attention models cache one row per token in ``k`` and nothing in ``v`` (value_dim 1 keeps the plumbing)
            v = torch.zeros_like(k) if dv == dk else torch.zeros((len(members), num_pages, heads, PAGE, dv), dtype=dtype,
                                                                 device=device)
            self.pools.append((k, v))
            self._kv_index.update({li: (g, i) for i, li in enumerate(members)})
        for li, donor in (donors or {}).items():
            self._kv_index[li] = self._kv_index[donor]
        self.pooled: dict = {}               # layer -> mean keys and values [pages, heads, blocks ending in a page, width]
        for li, block in (layer_pools or {}).items():
            k, v = self.layer(li)
            rows = -(-PAGE // block)
            self.pooled[li] = tuple(torch.zeros((*t.shape[:2], rows, t.shape[3]), dtype=dtype, device=device) for t in (k, v))
        self.k, self.v = self.pools[0]
        self._conv_index = {li: i for i, li in enumerate(conv_layers or [])}
        self.conv_state = None
        if self._conv_index:
            self.conv_state = torch.zeros((len(self._conv_index), num_pages, conv_hist, conv_channels), dtype=dtype,
                                          device=device)
        try:
            from ..lib import _eredu_host  # type: ignore

            self.allocator = _eredu_host.BlockManager(num_pages)
        except Exception:
            self.allocator = PageAllocator(num_pages)
        # Recurrent state of gated-delta layers: too large to keep per page, so sequences get a compact state slot and
        # `page_to_slot` (indexed by a sequence's first page, read on the device) finds it.
        self.la_conv_state = self.la_rec_state = self.page_to_slot = None
        self._la_index: dict = {}
        self.layer_state: dict = {}          # layer -> fp32 [slots, *shape] of families whose layers keep states of their own shape
        self._free_state_slots: list[int] = []
        self._slot_of_page: dict = {}

    def alloc(self, n: int) -> list:
        """Pages from the allocator. When lower tiers are attached (``block_tiers``), published pages that this
        allocation evicted are copied out at once - their contents are intact only until the new owner's first write."""
        pages = list(self.allocator.alloc(n))
        tiers = getattr(self, "block_tiers", None)
        if tiers is not None:
            tiers.demote(self.allocator.take_evicted())
        return pages

    def enable_linear_attention_state(self, layers, slots: int, conv_hist: int, conv_channels: int, heads: int, dk: int, dv: int):
        dev, dt = self.k.device, self.k.dtype
        self._la_index = {li: i for i, li in enumerate(layers)}
        n = len(self._la_index)
        self.la_conv_state = torch.zeros((n, slots, conv_hist, conv_channels), dtype=dt, device=dev)
        self.la_rec_state = torch.zeros((n, slots, heads, dk, dv), dtype=torch.float32, device=dev)
        self._make_slots(slots)

    def enable_layer_states(self, shapes: dict, slots: int):
        """fp32 recurrent states given per layer (``shapes``: layer -> shape of one sequence's state)."""
        dev = self.k.device
        self.layer_state = {li: torch.zeros((slots, *shape), dtype=torch.float32, device=dev) for li, shape in shapes.items()}
        self._make_slots(slots)

    def _make_slots(self, slots: int):
        self.page_to_slot = torch.zeros(self.num_pages, dtype=torch.int32, device=self.k.device)
        self._free_state_slots = list(range(slots - 1, -1, -1))
        self._slot_of_page = {}

    def bind_state(self, first_page: int) -> int:
        """Give the sequence that starts at ``first_page`` a zeroed state slot."""
        if self.page_to_slot is None:
            return -1
        if not self._free_state_slots:
            raise RuntimeError("KV pool exhausted (no free recurrent-state slot)")
        slot = self._free_state_slots.pop()
        self._slot_of_page[int(first_page)] = slot
        self.page_to_slot[int(first_page)] = slot
        for t in self._slot_views(slot):
            t.zero_()
        return slot

    def _slot_views(self, slot: int) -> list:
        """The recurrent state of one slot in every tensor that is indexed by slots."""
        views = [t[:, slot] for t in (self.la_conv_state, self.la_rec_state) if t is not None]
        return views + [t[slot] for t in self.layer_state.values()]

    def unbind_state(self, first_page: int) -> None:
        if self.page_to_slot is None:
            return
        slot = self._slot_of_page.pop(int(first_page), None)
        if slot is not None:
            self._free_state_slots.append(slot)

    def detach_state(self, first_page: int) -> int:
        """The sequence gives its pages up but keeps its state slot (parked in a host tier). Returns the slot or -1."""
        if self.page_to_slot is None:
            return -1
        return self._slot_of_page.pop(int(first_page), -1)

    def attach_state(self, slot: int, first_page: int) -> None:
        """A detached slot follows the sequence's new first page."""
        if self.page_to_slot is None or slot < 0:
            return
        self._slot_of_page[int(first_page)] = slot
        self.page_to_slot[int(first_page)] = slot

    def free_state_slot(self, slot: int) -> None:
        if self.page_to_slot is not None and slot >= 0:
            self._free_state_slots.append(slot)

    # ---- recurrent-state snapshots: K/V pages roll back by a length change, the fixed-size states of hybrid layers
    # (short-convolution history, gated-delta / Mamba matrices) have to be copied out and put back.
    def has_recurrent_state(self) -> bool:
        return self.conv_state is not None or self.page_to_slot is not None

    def recurrent_tensors(self) -> list:
        """Every fixed-size state tensor a forward pass mutates in place (empty for attention-only models). A step that
        is run twice on the same inputs - a warm-up before graph capture - must put these back in between: unlike a
        K/V append, advancing a recurrent state is not idempotent."""
        return [t for t in (self.conv_state, self.la_conv_state, self.la_rec_state, *self.layer_state.values()) if t is not None]

    def snapshot_state(self, first_page: int):
        """Copies of this sequence's recurrent states (None for attention-only models)."""
        if not self.has_recurrent_state():
            return None
        conv = self.conv_state[:, int(first_page)].clone() if self.conv_state is not None else None
        la = None
        if self.page_to_slot is not None:
            slot = self._slot_of_page[int(first_page)]
            la = tuple(t.clone() for t in self._slot_views(slot))
        return conv, la

    def restore_state(self, first_page: int, snap) -> None:
        if snap is None:
            return
        conv, la = snap
        if conv is not None:
            self.conv_state[:, int(first_page)].copy_(conv)
        if la is not None:
            slot = self._slot_of_page[int(first_page)]
            for t, saved in zip(self._slot_views(slot), la):
                t.copy_(saved)

    def linear_attention_state(self, li: int):
        i = self._la_index[li]
        return self.la_conv_state[i], self.la_rec_state[i]

    def layer(self, li: int):
        g, i = self._kv_index[li]
        k, v = self.pools[g]
        return k[i], v[i]

    def require_uniform(self, what: str) -> None:
        """Raised by the features that move pages of one geometry (lower tiers, parking)."""
        if len(self.pools) > 1:
            raise NotImplementedError(f"{what} needs one key / value geometry for all layers; this model has {len(self.pools)}")
        if self.pooled:
            raise NotImplementedError(f"{what} does not move pooled keys and values")

    def conv_layer(self, li: int):
        return self.conv_state[self._conv_index[li]]

    def bytes(self) -> int:
        extra = self.conv_state.numel() * self.conv_state.element_size() if self.conv_state is not None else 0
        if self.la_rec_state is not None:
            extra += self.la_rec_state.numel() * 4 + self.la_conv_state.numel() * self.la_conv_state.element_size()
        extra += sum(t.numel() * 4 for t in self.layer_state.values())
        pools = (*self.pools, *self.pooled.values())
        return sum((k.numel() + v.numel()) * k.element_size() for k, v in pools) + extra

    @staticmethod
    def pages_for(tokens: int) -> int:
        return (tokens + PAGE - 1) // PAGE
