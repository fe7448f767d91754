"""The cache's device storage: pages of keys and values per group, state per layer.

Layout of one group: [layer in group, K|V, page, kv head, token in page, head_dim];
a group whose values have another size than its keys holds two such tensors, one for
the keys and one, [..., value_dim], for the values.
A (page, kv head) tile is one contiguous [PAGE_TOKENS, head_dim] panel, so a kernel
streams whole panels and a 2-D bulk copy can fetch one.  State rows are float32
[slot, *state_shape] per layer and are zeroed when the slot is handed out; row number
`n_slots` belongs to no sequence and takes the padding rows of a fixed-size decode batch; a layer's block may keep
a second such area (`block_state`, [slot, n]).  Every group
has one page more than its pool hands out: page number `n_pages` belongs to no
sequence and takes the writes of the padding rows of a fixed-size decode batch.
A layer whose need says `pool` has a second pair of areas of the same layout, in a
group of their own, whose entries are blocks of that many tokens.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Dict, Optional, Sequence

import torch

from .book import PAGE_TOKENS, CacheBook, CacheNeed


@dataclass
class LayerCache:
    """What one layer's mixer gets: its pages (None: no keys) and its state rows (None: no state)."""
    group: Optional[int]
    keys: Optional[torch.Tensor]      # [n_pages, num_kv_heads, PAGE_TOKENS, head_dim]
    values: Optional[torch.Tensor]
    state: Optional[torch.Tensor]     # [n_slots, *state_shape] float32
    window: Optional[int] = None
    shared: bool = False              # the view of a layer that reads another layer's cache: it must not write
    block_state: Optional[torch.Tensor] = None   # [n_slots + 1, n] float32: what the layer's block keeps per sequence
    pool_group: Optional[int] = None             # the group of the pooled blocks, with their keys and values
    pool_keys: Optional[torch.Tensor] = None
    pool_values: Optional[torch.Tensor] = None


class KVCache(CacheBook):
    def __init__(self, needs: Sequence[Optional[CacheNeed]], max_tokens: int, max_seq_len: int,
                 dtype: torch.dtype, device, n_slots: Optional[int] = None, cache_from: Optional[Dict[int, int]] = None):
        super().__init__(needs, max_tokens, max_seq_len, n_slots)
        self.dtype, self.device = dtype, torch.device(device)
        self.stores = []          # per group: one tensor [layer, K|V, ...], or a (keys, values) pair of [layer, ...]
        for g in self.groups:
            shape = (g.n_pages + 1, g.need.num_kv_heads, PAGE_TOKENS)
            vd, nv = g.need.value_dim or g.need.head_dim, g.need.value_heads or g.need.num_kv_heads
            if vd == g.need.head_dim and nv == g.need.num_kv_heads:
                self.stores.append(torch.zeros((len(g.layers), 2) + shape + (vd,), dtype=dtype, device=self.device))
            else:
                self.stores.append((torch.zeros((len(g.layers),) + shape + (g.need.head_dim,), dtype=dtype, device=self.device),
                                    torch.zeros((len(g.layers), g.n_pages + 1, nv, PAGE_TOKENS, vd), dtype=dtype,
                                                device=self.device)))
        self.states = {layer: torch.zeros((self.n_slots + 1,) + shape, dtype=torch.float32, device=self.device)
                       for layer, shape in self.state_layers.items()}
        self.block_states = {layer: torch.zeros((self.n_slots + 1, n), dtype=torch.float32, device=self.device)
                             for layer, n in self.block_state_layers.items()}
        self._views: Dict[int, LayerCache] = {}
        for layer, need in enumerate(needs):
            if need is None:
                continue
            gi, pi = self.group_of_layer.get(layer), self.pool_group_of_layer.get(layer)
            keys, values = self._areas(gi, layer)
            pool_keys, pool_values = self._areas(pi, layer)
            self._views[layer] = LayerCache(gi, keys, values, self.states.get(layer),
                                            need.window if need.kind == "window" else None,
                                            block_state=self.block_states.get(layer),
                                            pool_group=pi, pool_keys=pool_keys, pool_values=pool_values)
        for layer, src in (cache_from or {}).items():
            self._views[layer] = dataclasses.replace(self._views[src], shared=True)

    def _areas(self, group: Optional[int], layer: int):
        """The keys and the values of `layer` in a group (None, None without one)."""
        if group is None:
            return None, None
        li, store = self.groups[group].layers.index(layer), self.stores[group]
        return (store[0][li], store[1][li]) if isinstance(store, tuple) else (store[li, 0], store[li, 1])

    def _on_alloc(self, slot: int) -> None:
        for state in list(self.states.values()) + list(self.block_states.values()):
            state[slot].zero_()

    def layer(self, index: int) -> LayerCache:
        return self._views[index]

    def bytes_per_token(self) -> int:
        item = torch.empty((), dtype=self.dtype).element_size()
        return sum(len(g.layers) * (g.need.num_kv_heads * g.need.head_dim
                                    + (g.need.value_heads or g.need.num_kv_heads) * (g.need.value_dim or g.need.head_dim)) * item
                   // (g.need.pool if g.pooled else 1) for g in self.groups)
