"""What the models built from the layer mechanisms share: weights padded to the kernels' row strides, the residual stream
walked sublayer by sublayer, the vocabulary projection, and the calls that ``Engine`` makes."""
from __future__ import annotations

from typing import Optional

import torch

from . import layer_ops, ops
from .layer_cache import LayeredKVManager
from .layer_ops import MoeSpec, pad8


class WeightPacker:
    """Checkpoint tensors -> device tensors whose sizes are padded with zeros to multiples of 8, group by group."""

    def __init__(self, weights, device, dtype):
        self.weights, self.device, self.dtype = weights, device, dtype

    def __getitem__(self, name):
        return self.weights[name]

    def zeros(self, *shape, dtype=None):
        return torch.zeros(*shape, dtype=dtype or self.dtype, device=self.device)

    def matrix(self, name, rows, cols):
        """`rows`, `cols`: (groups, size) or a size.  [groups * size, ...] -> [groups * pad8(size), ...]."""
        (gr, r), (gc, c) = (x if isinstance(x, tuple) else (1, x) for x in (rows, cols))
        t = self.weights[name]
        if tuple(t.shape) != (gr * r, gc * c):
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {(gr * r, gc * c)}")
        out = self.zeros(gr, pad8(r), gc, pad8(c))
        out[:, :r, :, :c] = t.view(gr, r, gc, c)
        return out.view(gr * pad8(r), gc * pad8(c))

    def vector(self, name, groups, size, to=torch.float32):
        t = self.weights[name]
        if t.numel() != groups * size:
            raise ValueError(f"{name}: {t.numel()} values, expected {groups * size}")
        out = self.zeros(groups, pad8(size), dtype=to)
        out[:, :size] = t.view(groups, size)
        return out.view(-1)

    def gate_up(self, gate, up, ff, cols):
        """[pad8(ff), 2, pad8(cols)]: the gate and the up row of every inner column."""
        return torch.stack((self.matrix(gate, ff, cols), self.matrix(up, ff, cols)), dim=1)

    def experts(self, prefix, spec: MoeSpec, bias: bool):
        """The tensors of a mixture of experts ('<prefix>e0.gate', ..., '<prefix>router')."""
        S, F = pad8(spec.width), pad8(spec.ff)
        gate_up, down = self.zeros(spec.experts, F, 2, S), self.zeros(spec.experts, S, F)
        for e in range(spec.experts):
            gate_up[e] = self.gate_up(f"{prefix}e{e}.gate", f"{prefix}e{e}.up", spec.ff, spec.width)
            down[e] = self.matrix(f"{prefix}e{e}.down", spec.width, spec.ff)
        router = self.zeros(spec.experts, S)
        t = self.weights[prefix + "router"]
        if tuple(t.shape) != (spec.experts, spec.width):
            raise ValueError(f"{prefix}router: shape {tuple(t.shape)}, expected {(spec.experts, spec.width)}")
        router[:, :spec.width] = t
        return dict(router=router, router_b=self.weights[prefix + "router.b"].float().to(self.device) if bias else None,
                    gate_up=gate_up, down=down, counts=self.zeros(spec.experts, dtype=torch.int32))


class LayeredModel:
    """Base of the models.  A subclass sets `cache_specs` (one per layer), `embed` [vocab, stride], and has
    ``_hidden(input_ids, batch_idx, kv)``: the normalised stream of every row, [rows, stride]."""

    def __init__(self, config, device, dtype):
        if dtype not in (torch.bfloat16, torch.float32):
            raise TypeError(f"{type(self).__name__} runs in bfloat16 or float32, not {dtype}")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        self.width, self.stride, self.eps = config.width, pad8(config.width), config.norm_eps
        self.status = ops.new_status(self.device)
        self.layers, self.cache_specs = [], []

    def new_cache(self, max_batch: int, max_seq_len: int, num_pages: Optional[int] = None, page_size: int = 64,
                  alias_layers: bool = False) -> LayeredKVManager:
        return LayeredKVManager(self.cache_specs, max_batch, max_seq_len, self.device, self.dtype, num_pages, page_size,
                                alias_layers)

    def _load_table(self, pack: WeightPacker) -> None:
        self.embed = pack.matrix("embed", self.config.vocab, self.width)[:self.config.vocab]

    # ---- parts of a forward
    def _stream(self, input_ids, center: bool = True):
        """(x, h, step): the residual stream, the buffer of a sublayer's input, and the row kernel over both (center: layer
        norms, else RMS norms)."""
        bsz, seq_len = input_ids.shape
        if bsz != 1 and seq_len != 1:
            raise ValueError(f"one sequence, or one token of each: input shape {tuple(input_ids.shape)}")
        x = torch.empty(bsz * seq_len, self.stride, dtype=torch.float32, device=self.device)
        h = torch.empty(bsz * seq_len, self.stride, dtype=self.dtype, device=self.device)

        def step(**kw):
            layer_ops.residual_norm(x, h, self.width, self.eps, center=center, status=self.status, **kw)
        return x, h, step

    def _experts(self, h, layer):
        """The weighted expert outputs of every row, [rows, top, stride]; the layer's counters have been cleared."""
        routing = layer_ops.moe_route(h, layer["router"], layer["router_b"], layer["moe"], layer["counts"])
        return layer_ops.moe_experts(h, layer["gate_up"], layer["down"], routing, layer["moe"], status=self.status)

    def _project(self, h):
        """fp32 products with the embedding table."""
        if self.dtype == torch.float32:
            return torch.mm(h, self.embed.t())
        return torch.mm(h, self.embed.t(), out_dtype=torch.float32)

    def _logits(self, h):
        return self._project(h)

    def _best(self, h):
        return self._project(h).argmax(dim=-1)

    # ---- what Engine calls
    @torch.no_grad()
    def inference(self, input_ids, position_ids, batch_idx, kv, rows=None):
        """input_ids [B, S] (one sequence's next S tokens, or one token of B sequences) -> fp32 logits [B, S, V].
        Positions are those of the cache (`position_ids` is what Engine passes to every model).  rows: project only
        these of the S tokens of a sequence, [1, len(rows), V]."""
        h = self._hidden(input_ids, batch_idx, kv)
        if rows is not None:
            h = h[torch.as_tensor(rows, dtype=torch.int64, device=h.device)]
            return self._logits(h).unsqueeze(0)
        return self._logits(h).view(*input_ids.shape, -1)

    @torch.no_grad()
    def next_tokens(self, input_ids, position_ids, batch_idx, kv, last_only: bool = False):
        """Greedy tokens of the rows (last_only: of the last row, a prompt's)."""
        h = self._hidden(input_ids, batch_idx, kv)
        return self._best(h[-1:] if last_only else h)

    def check_status(self):
        ops.raise_on_status(self.status)
