"""KV manager for models whose layers each have their own head sizes.

Pages come from the shared ``PagePool`` (``PooledTable`` keeps the slots, lengths and page tables); the cache of a
layer is two tensors, ``k_pages [pages, kv_heads * maps, page_size, dim]`` and ``v_pages [pages, kv_heads, page_size,
vdim]`` (a head's tokens of a page lie together: what one CTA reads is contiguous), sized by the layer's ``AttentionSpec``.  A layer hands over its fused projection rows (queries, keys and
values side by side): keys and values go from there into the pages, the attention kernel reads the queries in place.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from . import layer_ops, ops
from .engine import PooledTable


class LayeredKVManager(PooledTable):
    def __init__(self, specs: Sequence[layer_ops.AttentionSpec], max_batch_size: int, max_seq_len: int, device, dtype,
                 num_pages: Optional[int] = None, page_size: int = 64, alias_layers: bool = False):
        """specs: one per layer (a model's ``attention_specs``).  num_pages: pages of the pool, shared by all slots
        (None: max_seq_len tokens for every slot).  `alias_layers`: layers of equal sizes share one physical cache
        (a benchmark device, as in PooledKVManager)."""
        self.specs = list(specs)
        self.num_layers = len(self.specs)
        self.max_batch_size, self.max_length = max_batch_size, max_seq_len
        self.device, self.dtype = torch.device(device), dtype
        self.page_size = page_size
        self.pages_per_slot = (max_seq_len + page_size - 1) // page_size
        total = self.pages_per_slot * max_batch_size if num_pages is None else int(num_pages)
        self._init_table(total)
        shared = {}
        self.k_pages, self.v_pages = [], []
        for s in self.specs:
            shape = (s.kv_heads, s.maps, s.dim_stride, s.vdim_stride)
            if not alias_layers or shape not in shared:
                zeros = lambda heads, cols: torch.zeros(total, heads, page_size, cols, device=self.device, dtype=dtype)
                shared[shape] = (zeros(s.kv_heads * s.maps, s.dim_stride), zeros(s.kv_heads, s.vdim_stride))
            self.k_pages.append(shared[shape][0])
            self.v_pages.append(shared[shape][1])
        self.status = ops.new_status(self.device)
        self._workspace = None

    # ---- attention of one layer over the step's tokens
    def attend(self, proj: torch.Tensor, layer_idx: int, batch_idx: torch.Tensor, seq_len: int) -> torch.Tensor:
        """proj [rows, q | k | v columns]: one token of every slot of batch_idx (seq_len 1), or the next seq_len
        tokens of one slot.  Appends keys and values, returns the attention output [rows, heads * vdim]."""
        spec = self.specs[layer_idx]
        if self._step_table is not None:
            indices, indptr, last, _ = self._step_table      # prepare_step advanced the lengths
            slots = self._active
        else:
            slots = self._slots_of(batch_idx)
            lengths = [int(self._host_len[layer_idx][s]) + seq_len for s in slots]
            indices, indptr, last, _ = self._table_for(slots, lengths)
            for s in slots:
                self._host_len[layer_idx][s] += seq_len
        table = layer_ops.PageTable(indices, indptr, last, self.page_size, self._num_pool_pages)
        new_indptr = None
        if seq_len > 1:
            if len(slots) != 1:
                raise ValueError("several tokens at once: one sequence at a time")
            new_indptr = self._new_indptr(seq_len)
        k, v = self.k_pages[layer_idx], self.v_pages[layer_idx]
        layer_ops.kv_append(proj, spec.q_cols, spec.q_cols + spec.k_cols, k, v, table, spec, new_indptr,
                            status=self.status)
        splits = 1
        if new_indptr is None:
            longest = int(self._host_len[layer_idx][slots].max())
            splits = layer_ops.attention_splits(spec, len(slots), 1 << (longest - 1).bit_length(), self.dtype)
            need = layer_ops.attention_workspace(spec, len(slots), splits, self.dtype)
            if need and (self._workspace is None or self._workspace.numel() < need):
                self._workspace = torch.empty(need, dtype=torch.uint8, device=self.device)
        return layer_ops.paged_attention(proj, k, v, table, spec, new_indptr, seq_len, splits, self._workspace,
                                         status=self.status)

    def _new_indptr(self, seq_len: int) -> torch.Tensor:
        cached = getattr(self, "_indptr_of", None)
        if cached is None or cached[0] != seq_len:
            cached = self._indptr_of = (seq_len, torch.tensor([0, seq_len], dtype=torch.int32, device=self.device))
        return cached[1]

    def clear_cache(self, slot: int) -> None:
        """Give the slot's pages back (their contents are not read behind a sequence's length)."""
        self._release_slot(slot)

    def assume_filled(self, lengths: dict, headroom: int = 0) -> None:
        """Benchmark set-up: slot -> tokens its pages are taken to hold already, with room for `headroom` more."""
        for s in sorted(lengths):
            self.pool.admit(s, lengths[s], min(lengths[s] + headroom, self.max_length))
            self._host_len[:, s] = lengths[s]

    def check_status(self) -> None:
        ops.raise_on_status(self.status)
