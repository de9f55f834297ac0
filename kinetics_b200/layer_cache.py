"""Cache manager for models whose layers each have their own mixer and sizes.

Pages come from the shared ``PagePool`` (``PooledTable`` keeps the slots, lengths and page tables).  What a layer keeps
follows from its spec:

* ``AttentionSpec``: ``k_pages [pages, kv_heads * maps, page_size, dim]`` and ``v_pages [pages, kv_heads, page_size,
  vdim]`` (a head's tokens of a page lie together: what one CTA reads is contiguous);
* ``LatentSpec``: one row per token for all heads, ``k_pages [pages, 1, page_size, latent | rotated key]``, or the rows of
  the layer that `kv_from` names;
* ``LruSpec``: per slot an fp32 state and the newest inputs of the convolution.  A sequence that starts reads neither, so
  a slot that is used again needs no clearing.

A layer hands over its fused projection rows; the kernels read their columns in place.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from . import layer_ops, ops
from .engine import PooledTable


EXPAND_ROWS = 64        # from this many new tokens on, keys and values are expanded from the latents


def _rounded_up(n: int) -> int:
    """n to four leading bits, upwards: lengths that grow token by token change a launch's shape rarely."""
    step = 1 << max(n.bit_length() - 4, 0)
    return (n + step - 1) // step * step


@dataclass
class LatentWeights:
    """What a latent-attention layer brings to the manager: expansions of the latent to every head's keys
    uk [heads, dim, rank] and values uv [heads, vdim, rank] (padded sizes; both views of ukv [heads * (dim + vdim), rank]),
    sinks fp32 [heads], the latent's norm fp32 [rank] (None with kv_from), turns per position fp64 [rot_dim / 2]."""
    ukv: torch.Tensor
    uk: torch.Tensor
    uv: torch.Tensor
    sink: torch.Tensor
    norm: Optional[torch.Tensor]
    turns: torch.Tensor


@dataclass
class LruWeights:
    """conv_w fp32 [taps, cols], gates [blocks, 2 * block, block], the rest fp32 [cols]; decay = the factor of -r in log a."""
    conv_w: torch.Tensor
    conv_b: torch.Tensor
    gates: torch.Tensor
    rb: torch.Tensor
    ib: torch.Tensor
    decay: torch.Tensor


@dataclass
class LayerStep:
    """One layer's call: the page table after the step, rows per sequence (None: one each), slots on the device."""
    table: layer_ops.PageTable
    new_indptr: Optional[torch.Tensor]
    slots: torch.Tensor
    sequences: int
    longest: int


class LayeredKVManager(PooledTable):
    def __init__(self, specs: Sequence, max_batch_size: int, max_seq_len: int, device, dtype,
                 num_pages: Optional[int] = None, page_size: int = 64, alias_layers: bool = False):
        """specs: one per layer (a model's ``cache_specs``).  num_pages: pages of the pool, shared by all slots
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
        self.k_pages, self.v_pages, self.states, self.rings = [], [], [], []
        zeros = lambda heads, cols: torch.zeros(total, heads, page_size, cols, device=self.device, dtype=dtype)
        for i, s in enumerate(self.specs):
            k = v = state = ring = None
            if isinstance(s, layer_ops.LruSpec):
                state = torch.zeros(max_batch_size, s.cols, device=self.device)
                ring = torch.zeros(max_batch_size, s.taps, s.cols, device=self.device, dtype=dtype)
            elif isinstance(s, layer_ops.LatentSpec) and s.kv_from is not None:
                k = v = self.k_pages[s.kv_from]
            else:
                latent = isinstance(s, layer_ops.LatentSpec)
                shape = s.row_cols if latent else (s.kv_heads, s.maps, s.dim_stride, s.vdim_stride)
                if not alias_layers or shape not in shared:
                    shared[shape] = (zeros(1, s.row_cols),) * 2 if latent else \
                        (zeros(s.kv_heads * s.maps, s.dim_stride), zeros(s.kv_heads, s.vdim_stride))
                k, v = shared[shape]
            self.k_pages.append(k)
            self.v_pages.append(v)
            self.states.append(state)
            self.rings.append(ring)
        self.status = ops.new_status(self.device)
        self._workspace = None

    def _view(self, slots, order=None):
        return slots                                         # the slots of the step's sequences, on the device

    def _step_of(self, layer_idx: int, batch_idx: torch.Tensor, seq_len: int) -> LayerStep:
        """Advances the layer by one token of every slot of batch_idx (seq_len 1), or by seq_len tokens of one slot."""
        if self._step_table is not None:
            indices, indptr, last, slots_dev = self._step_table      # prepare_step advanced the lengths
            slots = self._active
        else:
            slots = self._slots_of(batch_idx)
            lengths = [int(self._host_len[layer_idx][s]) + seq_len for s in slots]
            indices, indptr, last, slots_dev = self._table_for(slots, lengths)
            for s in slots:
                self._host_len[layer_idx][s] += seq_len
        table = layer_ops.PageTable(indices, indptr, last, self.page_size, self._num_pool_pages)
        new_indptr = None
        if seq_len > 1:
            if len(slots) != 1:
                raise ValueError("several tokens at once: one sequence at a time")
            new_indptr = self._new_indptr(seq_len)
        return LayerStep(table, new_indptr, slots_dev, len(slots), int(self._host_len[layer_idx][slots].max()))

    def _attention(self, q, k, v, step: LayerStep, spec: layer_ops.AttentionSpec, seq_len: int, **kw) -> torch.Tensor:
        splits = layer_ops.attention_splits(spec, step.sequences, _rounded_up(step.longest), self.dtype,
                                            0 if step.new_indptr is None else seq_len)
        need = layer_ops.attention_workspace(spec, q.shape[0], splits, self.dtype)
        if need and (self._workspace is None or self._workspace.numel() < need):
            self._workspace = torch.empty(need, dtype=torch.uint8, device=self.device)
        return layer_ops.paged_attention(q, k, v, step.table, spec, step.new_indptr, seq_len, splits, self._workspace,
                                         status=self.status, **kw)

    # ---- the mixers of one layer over the step's tokens: proj [rows, the columns of the layer's spec]
    def attend(self, proj: torch.Tensor, layer_idx: int, batch_idx: torch.Tensor, seq_len: int) -> torch.Tensor:
        """proj [rows, q | k | v columns]: appends keys and values, returns the attention output [rows, heads * vdim]."""
        spec = self.specs[layer_idx]
        step = self._step_of(layer_idx, batch_idx, seq_len)
        k, v = self.k_pages[layer_idx], self.v_pages[layer_idx]
        layer_ops.kv_append(proj, spec.q_cols, spec.q_cols + spec.k_cols, k, v, step.table, spec, step.new_indptr,
                            status=self.status)
        return self._attention(proj, k, v, step, spec, seq_len)

    def attend_latent(self, proj: torch.Tensor, layer_idx: int, batch_idx: torch.Tensor, seq_len: int,
                      w: LatentWeights) -> torch.Tensor:
        """proj [rows, q | latent, rotated key | gates]: appends the latents (unless the layer reads another's), returns
        the gated attention output [rows, heads * vdim].  A decode step and a short portion: the queries take the key
        expansion, q uk, and the heads' values are expanded behind the attention, so that per token only the latent row is
        read.  A long portion: keys and values of the whole sequence are expanded first, which is less arithmetic per
        query."""
        spec = self.specs[layer_idx]
        step = self._step_of(layer_idx, batch_idx, seq_len)
        rows, H, pages = proj.shape[0], spec.heads, self.k_pages[layer_idx]
        gate = proj[:, spec.gate_col:]
        dim, rank, vdim = w.uk.shape[1], w.uk.shape[2], w.uv.shape[1]
        if rows >= EXPAND_ROWS and step.new_indptr is not None and layer_ops.expanded_supported(spec, self.dtype):
            layer_ops.latent_append(proj, spec, step.table, pages, w.norm, w.turns, step.new_indptr, status=self.status)
            latents = layer_ops.gather_rows(pages, step.table, step.longest, status=self.status)
            kv = torch.mm(latents[:, :rank], w.ukv.t())
            return layer_ops.expanded_attention(proj, kv, latents, spec, w.sink, gate, status=self.status)
        q = torch.empty(rows, H, spec.row_cols, dtype=proj.dtype, device=proj.device)
        layer_ops.latent_append(proj, spec, step.table, pages, w.norm, w.turns, step.new_indptr, q, status=self.status)
        heads = proj[:, :spec.q_cols].view(rows, H, -1)
        torch.bmm(heads[:, :, :dim].transpose(0, 1), w.uk, out=q[:, :, :rank].transpose(0, 1))
        latent = self._attention(q.view(rows, -1), pages, pages, step, spec.rows(), seq_len, sink=w.sink, gate=gate)
        out = torch.empty(rows, H, vdim, dtype=proj.dtype, device=proj.device)
        torch.bmm(latent.view(rows, H, rank).transpose(0, 1), w.uv.transpose(1, 2), out=out.transpose(0, 1))
        return out.view(rows, -1)

    def recur(self, proj: torch.Tensor, layer_idx: int, batch_idx: torch.Tensor, seq_len: int, w: LruWeights) -> torch.Tensor:
        """proj [rows, y | x]: advances the slots' convolution and state, returns the gated state [rows, cols]."""
        spec, step = self.specs[layer_idx], self._step_of(layer_idx, batch_idx, seq_len)
        if step.new_indptr is None and layer_ops.lru_decode_supported(spec, self.dtype):
            return layer_ops.lru_decode(proj, spec, step.table, step.slots, w.conv_w, w.conv_b, w.gates, w.rb, w.ib, w.decay,
                                        self.rings[layer_idx], self.states[layer_idx], status=self.status)
        run = dict(new_indptr=step.new_indptr, max_new=seq_len, status=self.status)
        u = layer_ops.lru_conv(proj, spec, step.table, step.slots, w.conv_w, w.conv_b, self.rings[layer_idx], **run)
        z = layer_ops.lru_gate_products(u, w.gates, spec)
        return layer_ops.lru_scan(z, u, proj, spec, step.table, step.slots, w.rb, w.ib, w.decay, self.states[layer_idx],
                                  **run)

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
