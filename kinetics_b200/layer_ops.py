"""Wrappers of libktk_layers.so (``include/ktk_layers.h``): layer mechanisms whose sizes and constants are parameters.

Every call runs a hand-written CUDA kernel on the current stream; a CPU tensor raises.  ``variant`` picks a kernel
(``VARIANT_AUTO``: the fastest built one for the sizes); the fp32 forms and odd sizes run on the FMA kernels.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from ._lib import VARIANT_AUTO, check_layers
from .ops import _cuda, _dtype_code, _launched, _ptr, _stream

MAX_EXPERTS = 1024


def pad8(n: int) -> int:
    """Columns in memory of a row of n: the next multiple of 8 (the rest holds zeros)."""
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class AttentionSpec:
    """One layer's attention over its paged cache.

    maps = 1: softmax(scores) v.  maps = 2: every head has two score maps over the same values; the output is their
    difference a1 - lam a2, divided by sqrt(mean square + eps) and multiplied by out_scale.  A score is
    (q . k) * scale times the query's temperature 1 + temp_coef ln(floor((position + 1) / temp_every) + 1), then
    softcap tanh(score / softcap) if softcap > 0.  values_in_keys: the value of a token is the first vdim columns of
    its key row (one tensor holds both)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    maps: int = 1
    softcap: float = 0.0
    temp_coef: float = 0.0
    temp_every: float = 1.0
    lam: float = 0.0
    eps: float = 1e-6
    out_scale: float = 1.0
    values_in_keys: bool = False

    @property
    def dim_stride(self) -> int:
        return pad8(self.dim)

    @property
    def vdim_stride(self) -> int:
        return pad8(self.vdim)

    @property
    def q_cols(self) -> int:
        return self.heads * self.maps * self.dim_stride

    @property
    def k_cols(self) -> int:
        return self.kv_heads * self.maps * self.dim_stride

    @property
    def v_cols(self) -> int:
        return self.kv_heads * self.vdim_stride

    @property
    def o_cols(self) -> int:
        return self.heads * self.vdim_stride

    def c(self, dtype_code: int) -> _lib.Attn:
        return _lib.Attn(self.heads, self.kv_heads, self.maps, self.dim, self.vdim, self.dim_stride, self.vdim_stride,
                         dtype_code, self.scale, self.softcap, self.temp_coef, self.temp_every, self.lam, self.eps,
                         self.out_scale, self.dim_stride if self.values_in_keys else 0)


@dataclass(frozen=True)
class GateSpec:
    """Gated activation g' sigmoid(slope g') (u' + shift), g' = min(g, limit), u' = clamp(u, -limit, limit)."""
    limit: float = math.inf
    slope: float = 1.0
    shift: float = 0.0


SILU = GateSpec()


@dataclass(frozen=True)
class MoeSpec:
    """A mixture of experts: each row uses the `top` of `experts` gated feed-forwards of inner size ff.  Weights: the
    softmax over the chosen logits, or (score_all) the chosen ones' share of the softmax over all."""
    experts: int
    top: int
    width: int
    ff: int
    score_all: bool = False
    gate: "GateSpec" = SILU

    def c(self, dtype_code: int) -> _lib.Moe:
        return _lib.Moe(self.experts, self.top, self.width, self.ff, pad8(self.width), pad8(self.ff), dtype_code,
                        int(self.score_all), self.gate.limit, self.gate.slope, self.gate.shift)


@dataclass(frozen=True)
class Rotation:
    """Rotary positions on pairs (2 i, 2 i + 1) of `dims` columns: base^(-2 i / dims) radians per position, and with
    factor != 1 their stretch for contexts beyond `original` (YaRN): pairs that turn at least `fast` times within
    `original` positions keep their frequency, those that turn less than `slow` times have it divided by factor, a ramp
    in between; cos and sin are multiplied by 0.1 ln(factor) + 1."""
    dims: int
    base: float
    factor: float = 1.0
    original: float = 1.0
    fast: float = 1.0
    slow: float = 1.0
    scaled: bool = False

    def frequencies(self) -> torch.Tensor:
        """Radians per position, fp64 [dims / 2]."""
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = self.base ** (-2.0 * i / self.dims)
        if self.scaled:
            pair_of = lambda turns: self.dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(self.base))
            lo = max(math.floor(pair_of(self.fast)), 0)
            hi = min(math.ceil(pair_of(self.slow)), self.dims - 1)
            stretched = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
            f = torch.lerp(f, f / self.factor, stretched)
        return f

    def turns(self) -> torch.Tensor:
        """Whole turns per position, fp64 [dims / 2]: what latent_append takes."""
        return self.frequencies() / (2 * math.pi)

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0 if self.scaled else 1.0


@dataclass(frozen=True)
class LatentSpec:
    """Attention whose heads expand their keys and values from one cached latent per token, beside one rotated key part
    that all heads share.  Columns of a layer's projection rows: queries (heads of [dim | rot_dim]), the latent and the
    rotated key (unless kv_from names the layer whose cached rows are read), the output gates."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    rank: int
    scale: float
    rotation: Rotation
    eps: float = 1e-6
    kv_from: Optional[int] = None

    @property
    def row_cols(self) -> int:
        """Columns of a cached row."""
        return pad8(self.rank) + pad8(self.rot_dim)

    @property
    def head_cols(self) -> int:
        return pad8(self.dim) + pad8(self.rot_dim)

    @property
    def q_cols(self) -> int:
        return self.heads * self.head_cols

    @property
    def gate_col(self) -> int:
        return self.q_cols + (self.row_cols if self.kv_from is None else 0)

    @property
    def proj_cols(self) -> int:
        return self.gate_col + pad8(self.heads)

    def rows(self) -> AttentionSpec:
        """The attention over the cached rows, by queries that carry the key expansion."""
        return AttentionSpec(heads=self.heads, kv_heads=1, dim=self.row_cols, vdim=self.rank, scale=self.scale,
                             values_in_keys=True)

    def c(self, dtype_code: int) -> _lib.Latent:
        return _lib.Latent(self.heads, self.dim, self.rot_dim, self.vdim, self.rank, pad8(self.dim), pad8(self.rot_dim),
                           pad8(self.vdim), pad8(self.rank), dtype_code, self.scale, self.eps, self.rotation.amplitude)


@dataclass(frozen=True)
class LruSpec:
    """A linear recurrence with real gates behind a causal convolution of `taps` tokens: `blocks` blocks of `block`
    channels (see ``ktk_lru``).  Columns of a layer's projection rows: the output branch y, the recurrence's input x."""
    blocks: int
    block: int
    taps: int

    @property
    def cols(self) -> int:
        return self.blocks * pad8(self.block)

    def c(self, dtype_code: int) -> _lib.Lru:
        return _lib.Lru(self.blocks, self.block, pad8(self.block), self.taps, dtype_code)


class PageTable:
    """CSR page table of a step on the device (int32): see ``ktk_paged``."""

    def __init__(self, kv_indices, kv_indptr, kv_last_page_len, page_size: int, num_pages: int):
        for t in (kv_indices, kv_indptr, kv_last_page_len):
            _cuda(t)
            if t.dtype != torch.int32:
                raise TypeError("page tables are int32")
        self.tensors = (kv_indices, kv_indptr, kv_last_page_len)
        self.batch = kv_indptr.numel() - 1
        if kv_last_page_len.numel() != self.batch:
            raise ValueError("kv_last_page_len must have one entry per sequence")
        self.page_size, self.num_pages = page_size, num_pages

    def c(self) -> _lib.Paged:
        i, p, l = self.tensors
        return _lib.Paged(i.data_ptr(), p.data_ptr(), l.data_ptr(), self.batch, self.page_size, self.num_pages)


def residual_norm(x, h, cols: int, eps: float, pre=None, y=None, parts: int = 1, post=None, mult: float = 1.0,
                  tokens=None, embed=None, embed_scale: float = 1.0, center: bool = True, zero=None, status=None) -> None:
    """Rows of the fp32 residual stream x [rows, stride], in place: x = embed[tokens] * embed_scale (if given); x +=
    mult * norm(sum of y [rows, parts, stride]; post) (if y is given; post None: no norm); h = norm(x; pre), or x itself
    (pre None), in the dtype of h (if h is given).  pre / post: (weight, bias or None), fp32 [stride].  zero: an int32 tensor to clear."""
    rows, stride = x.shape
    code = _dtype_code(h if h is not None else y if y is not None else embed)
    pw, pb = post if post is not None else (None, None)
    nw, nb = pre if pre is not None else (None, None)
    _cuda(x, h, y, pw, pb, nw, nb, tokens, embed, zero, status)
    if x.dtype != torch.float32 or any(t is not None and (t.dtype != torch.float32 or t.numel() != stride)
                                       for t in (pw, pb, nw, nb)):
        raise TypeError("residual_norm: x and the norm weights are fp32, as wide as the rows")
    if h is not None and tuple(h.shape) != (rows, stride) or y is not None and y.numel() != rows * parts * stride:
        raise ValueError("residual_norm: h [rows, stride], y [rows, parts, stride]")
    if y is not None and _dtype_code(y) != code or embed is not None and _dtype_code(embed) != code:
        raise TypeError("residual_norm: h, y and embed share a dtype")
    if tokens is not None and (tokens.dtype != torch.int64 or tokens.numel() != rows or embed.shape[1] != stride):
        raise ValueError("residual_norm: tokens int64 [rows], embed [vocab, stride]")
    check_layers(_lib.load_layers().ktk_residual_norm(
        _ptr(tokens), _ptr(embed), 0 if embed is None else embed.shape[0], embed_scale, _ptr(x), _ptr(y), parts, _ptr(pw), _ptr(pb),
        mult, _ptr(nw), _ptr(nb), _ptr(h), eps, int(center), rows, cols, stride, _ptr(zero),
        0 if zero is None else zero.numel(), code, _ptr(status), _stream()))
    _launched()


def _cache_check(spec: AttentionSpec, table: PageTable, k_pages, v_pages):
    v_cols = spec.dim_stride if spec.values_in_keys else spec.vdim_stride
    if tuple(k_pages.shape) != (table.num_pages, spec.kv_heads * spec.maps, table.page_size, spec.dim_stride) or \
            tuple(v_pages.shape) != (table.num_pages, spec.kv_heads, table.page_size, v_cols):
        raise ValueError(f"cache shapes {tuple(k_pages.shape)}, {tuple(v_pages.shape)} do not fit {spec}")


def kv_append(proj, k_col: int, v_col: int, k_pages, v_pages, table: PageTable, spec: AttentionSpec, new_indptr=None,
              status=None) -> None:
    """Keys and values out of rows of proj [rows, cols] into their pages (the table already includes them)."""
    _cuda(proj, k_pages, v_pages, new_indptr, status)
    _cache_check(spec, table, k_pages, v_pages)
    a, t = spec.c(_dtype_code(k_pages)), table.c()
    if proj.dtype != k_pages.dtype or v_pages.dtype != k_pages.dtype:
        raise TypeError("kv_append: proj and the cache share a dtype")
    check_layers(_lib.load_layers().ktk_kv_append(_ptr(proj), proj.shape[1], k_col, v_col, _ptr(new_indptr),
                                                  proj.shape[0], _ptr(k_pages), _ptr(v_pages), ctypes.byref(t),
                                                  ctypes.byref(a), _ptr(status), _stream()))
    _launched()


def attention_splits(spec: AttentionSpec, batch: int, max_keys: int, dtype, new_rows: int = 0) -> int:
    a = spec.c(_lib.KTK_BF16 if dtype == torch.bfloat16 else _lib.KTK_F32)
    return int(_lib.load_layers().ktk_paged_attention_splits(ctypes.byref(a), batch, new_rows, max_keys))


def attention_workspace(spec: AttentionSpec, rows: int, splits: int, dtype) -> int:
    a = spec.c(_lib.KTK_BF16 if dtype == torch.bfloat16 else _lib.KTK_F32)
    return int(_lib.load_layers().ktk_paged_attention_workspace(ctypes.byref(a), rows, splits))


def paged_attention(proj, k_pages, v_pages, table: PageTable, spec: AttentionSpec, new_indptr=None, max_new: int = 1,
                    splits: int = 1, workspace=None, variant: int = VARIANT_AUTO, out=None, status=None, sink=None,
                    gate=None):
    """Causal attention of the rows of proj (whose first spec.q_cols columns are the queries) over their sequences;
    their keys are already in the pages.  new_indptr int32 [batch + 1]: rows per sequence; None: one each.
    sink fp32 [heads]: exp(sink) joins every denominator; gate [rows, >= heads] (a column range of a wider tensor is
    fine): head h of a row is multiplied by sigmoid(gate[row, h]).  Returns [rows, heads * vdim_stride]."""
    _cuda(proj, k_pages, v_pages, new_indptr, workspace, out, status, sink)
    if gate is not None and (gate.dtype != proj.dtype or gate.shape[0] != proj.shape[0] or gate.stride(1) != 1) or \
            sink is not None and (sink.dtype != torch.float32 or sink.numel() != spec.heads):
        raise ValueError("paged_attention: sink fp32 [heads], gate [rows, heads] in the dtype of the queries")
    _cache_check(spec, table, k_pages, v_pages)
    if proj.dtype != k_pages.dtype or v_pages.dtype != k_pages.dtype:
        raise TypeError("paged_attention: proj and the cache share a dtype")
    a, t = spec.c(_dtype_code(k_pages)), table.c()
    rows = proj.shape[0]
    if out is None:
        out = torch.empty(rows, spec.o_cols, dtype=proj.dtype, device=proj.device)
    if splits > 1 and workspace is None:
        need = attention_workspace(spec, rows, splits, proj.dtype)
        if need:
            workspace = torch.empty(need, dtype=torch.uint8, device=proj.device)
    wsb = 0 if workspace is None else workspace.numel()
    check_layers(_lib.load_layers().ktk_paged_attention(
        _ptr(proj), proj.shape[1], _ptr(new_indptr), rows, max_new, _ptr(k_pages), _ptr(v_pages), ctypes.byref(t),
        _ptr(sink), None if gate is None else gate.data_ptr(), 0 if gate is None else gate.stride(0), _ptr(out),
        _ptr(workspace), wsb, splits, variant, ctypes.byref(a), _ptr(status), _stream()))
    _launched(2 if splits > 1 else 1)
    return out


class Routing:
    """Where the rows of a step go: ids / weights [rows, top], counts [experts], bucket [experts, rows]."""

    def __init__(self, spec: MoeSpec, rows: int, device, counts: Optional[torch.Tensor] = None):
        self.ids = torch.empty(rows, spec.top, dtype=torch.int32, device=device)
        self.weights = torch.empty(rows, spec.top, dtype=torch.float32, device=device)
        self.counts = counts if counts is not None else torch.zeros(spec.experts, dtype=torch.int32, device=device)
        self.bucket = torch.empty(spec.experts, rows, dtype=torch.int32, device=device)


def moe_route(h, w, b, spec: MoeSpec, counts=None, variant: int = VARIANT_AUTO) -> Routing:
    """Router of rows h [rows, pad8(width)]: w [experts, pad8(width)] in the dtype of h, b fp32 [experts] or None.  counts:
    a cleared int32 [experts] tensor to count into (None: a new one)."""
    _cuda(h, w, b, counts)
    if w.dtype != h.dtype or b is not None and b.dtype != torch.float32 or tuple(w.shape) != (spec.experts, h.shape[1]):
        raise ValueError("moe_route: w [experts, row stride] in the dtype of h, b fp32")
    r = Routing(spec, h.shape[0], h.device, counts)
    m = spec.c(_dtype_code(h))
    check_layers(_lib.load_layers().ktk_moe_route(_ptr(h), _ptr(w), _ptr(b), _ptr(r.ids), _ptr(r.weights),
                                                  _ptr(r.counts), _ptr(r.bucket), h.shape[0], ctypes.byref(m), variant,
                                                  _stream()))
    _launched()
    return r


def moe_experts(h, gate_up, down, routing: Routing, spec: MoeSpec, variant: int = VARIANT_AUTO, status=None):
    """The chosen experts' weighted outputs [rows, top, pad8(width)] (their sum over `top` is the layer's output;
    residual_norm takes it with parts = top).  gate_up [experts, pad8(ff), 2, pad8(width)] (the gate and
    the up row of each inner column), down [experts, pad8(width), pad8(ff)]."""
    _cuda(h, gate_up, down, status)
    rows, ws = h.shape
    fs = pad8(spec.ff)
    if tuple(gate_up.shape) != (spec.experts, fs, 2, ws) or tuple(down.shape) != (spec.experts, ws, fs) or \
            gate_up.dtype != h.dtype or down.dtype != h.dtype:
        raise ValueError("moe_experts: gate_up [experts, ff stride, 2, row stride], down [experts, row stride, ff stride]")
    m = spec.c(_dtype_code(h))
    act = torch.empty(rows * spec.top, fs, dtype=h.dtype, device=h.device)
    y = torch.empty(rows, spec.top, ws, dtype=h.dtype, device=h.device)
    lib = _lib.load_layers()
    for stage, src, w, dst in ((0, h, gate_up, act), (1, act, down, y)):
        check_layers(lib.ktk_moe_gemm(stage, _ptr(src), _ptr(w), _ptr(dst), _ptr(routing.weights),
                                      _ptr(routing.counts), _ptr(routing.bucket), rows, ctypes.byref(m), variant,
                                      _ptr(status), _stream()))
        _launched()
    return y


def gated_rows(x, gate: GateSpec = SILU):
    """x [rows, 2 * cols] (gate columns, then up columns) -> gated activation [rows, cols]."""
    _cuda(x)
    rows, cols = x.shape[0], x.shape[1] // 2
    out = torch.empty(rows, cols, dtype=x.dtype, device=x.device)
    check_layers(_lib.load_layers().ktk_gated_rows(_ptr(x), _ptr(out), rows, cols, gate.limit, gate.slope, gate.shift,
                                                   _dtype_code(x), _stream()))
    _launched()
    return out


def scale_cap(z, scale: float, cap: float):
    """fp32 z <- cap tanh(z scale / cap), in place (cap 0: z scale)."""
    _cuda(z)
    if z.dtype != torch.float32:
        raise TypeError("scale_cap: fp32")
    check_layers(_lib.load_layers().ktk_scale_cap(_ptr(z), z.numel(), scale, cap, _stream()))
    _launched()
    return z


def latent_append(proj, spec: LatentSpec, table: PageTable, pages, norm_w, turns, new_indptr=None, q_out=None,
                  status=None) -> None:
    """Turns the queries' rotated parts (into q_out [rows, heads, row_cols], or in place) and, where the layer has its
    own, writes normalised latents and rotated keys to their page rows (the table already includes them)."""
    _cuda(proj, pages, norm_w, turns, new_indptr, q_out, status)
    if proj.dtype != pages.dtype or q_out is not None and q_out.dtype != proj.dtype or turns.dtype != torch.float64 or \
            norm_w is not None and norm_w.dtype != torch.float32:
        raise TypeError("latent_append: proj, q_out and the cache share a dtype; the norm is fp32, turns fp64")
    if proj.shape[1] != spec.proj_cols or turns.numel() != spec.rot_dim // 2 or \
            tuple(pages.shape) != (table.num_pages, 1, table.page_size, spec.row_cols) or \
            q_out is not None and tuple(q_out.shape) != (proj.shape[0], spec.heads, spec.row_cols):
        raise ValueError(f"latent_append: shapes {tuple(proj.shape)}, {tuple(pages.shape)} do not fit {spec}")
    own = spec.kv_from is None
    a, t = spec.c(_dtype_code(proj)), table.c()
    check_layers(_lib.load_layers().ktk_latent_append(
        _ptr(proj), proj.shape[1], 0, spec.q_cols if own else -1, _ptr(new_indptr), proj.shape[0],
        _ptr(norm_w if own else None), _ptr(turns), _ptr(q_out), _ptr(pages), ctypes.byref(t), ctypes.byref(a), _ptr(status),
        _stream()))
    _launched()


def gather_rows(pages, table: PageTable, total: int, status=None):
    """The first `total` rows of the table's only sequence, in order: pages [pages, 1, page_size, cols] -> [total, cols]."""
    _cuda(pages, status)
    out = torch.empty(total, pages.shape[-1], dtype=pages.dtype, device=pages.device)
    t = table.c()
    check_layers(_lib.load_layers().ktk_gather_rows(_ptr(pages), _ptr(out), total, pages.shape[-1] * pages.element_size(),
                                                    ctypes.byref(t), _ptr(status), _stream()))
    _launched()
    return out


def expanded_supported(spec: LatentSpec, dtype) -> bool:
    a = spec.c(_lib.KTK_BF16 if dtype == torch.bfloat16 else _lib.KTK_F32)
    return bool(_lib.load_layers().ktk_expanded_attention_supported(ctypes.byref(a)))


def expanded_attention(proj, kv, latents, spec: LatentSpec, sink=None, gate=None, status=None):
    """The newest rows of a sequence (proj, whose first columns are the rotated queries) over kv [total, keys of all heads |
    values of all heads], expanded from latents [total, row_cols] -> [rows, heads * pad8(vdim)]."""
    _cuda(proj, kv, latents, sink, status)
    rows, total, H = proj.shape[0], latents.shape[0], spec.heads
    if tuple(kv.shape) != (total, H * (pad8(spec.dim) + pad8(spec.vdim))) or latents.shape[1] != spec.row_cols or \
            any(t.dtype != torch.bfloat16 for t in (proj, kv, latents)):
        raise ValueError(f"expanded_attention: shapes {tuple(kv.shape)}, {tuple(latents.shape)} do not fit {spec}")
    out = torch.empty(rows, H * pad8(spec.vdim), dtype=proj.dtype, device=proj.device)
    a = spec.c(_lib.KTK_BF16)
    check_layers(_lib.load_layers().ktk_expanded_attention(
        _ptr(proj), proj.stride(0), rows, total, _ptr(kv), _ptr(latents), _ptr(sink),
        None if gate is None else gate.data_ptr(), 0 if gate is None else gate.stride(0), _ptr(out), ctypes.byref(a),
        _ptr(status), _stream()))
    _launched()
    return out


def lru_conv(proj, spec: LruSpec, table: PageTable, slots, conv_w, conv_b, ring, new_indptr=None, max_new: int = 1,
             status=None):
    """The causal convolution of the x columns of proj [rows, 2 * cols] -> u [rows, cols]; updates the ring
    [slots, taps, cols] of the sequences' slots."""
    _cuda(proj, slots, conv_w, conv_b, ring, new_indptr, status)
    if proj.shape[1] != 2 * spec.cols or ring.dtype != proj.dtype or tuple(ring.shape[1:]) != (spec.taps, spec.cols) or \
            tuple(conv_w.shape) != (spec.taps, spec.cols) or conv_w.dtype != torch.float32 or \
            conv_b.dtype != torch.float32 or slots.dtype != torch.int32 or slots.numel() != table.batch:
        raise ValueError(f"lru_conv: shapes {tuple(proj.shape)}, {tuple(ring.shape)} do not fit {spec}")
    u = torch.empty(proj.shape[0], spec.cols, dtype=proj.dtype, device=proj.device)
    a, t = spec.c(_dtype_code(proj)), table.c()
    check_layers(_lib.load_layers().ktk_lru_conv(
        _ptr(proj), proj.shape[1], spec.cols, _ptr(new_indptr), proj.shape[0], max_new, _ptr(slots), ring.shape[0],
        _ptr(conv_w), _ptr(conv_b), _ptr(ring), _ptr(u), ctypes.byref(t), ctypes.byref(a), _ptr(status), _stream()))
    _launched()
    return u


def lru_gate_products(u, w, spec: LruSpec):
    """Block-diagonal products, fp32: u [rows, cols], w [blocks, 2 * block stride, block stride] (the rows of r, then of
    i) -> [blocks, rows, 2 * block stride]."""
    parts = u.view(u.shape[0], spec.blocks, -1).transpose(0, 1)
    if u.dtype == torch.float32:
        return torch.bmm(parts, w.transpose(1, 2))
    return torch.bmm(parts, w.transpose(1, 2), out_dtype=torch.float32)


def lru_scan(z, u, proj, spec: LruSpec, table: PageTable, slots, rb, ib, decay, state, new_indptr=None, max_new: int = 1,
             status=None):
    """Gates, recurrence and output gate: z as lru_gate_products gives it, the y columns of proj -> [rows, cols];
    updates state fp32 [slots, cols]."""
    _cuda(z, u, proj, slots, rb, ib, decay, state, new_indptr, status)
    rows = proj.shape[0]
    if tuple(z.shape) != (spec.blocks, rows, 2 * pad8(spec.block)) or z.dtype != torch.float32 or \
            state.dtype != torch.float32 or state.shape[1] != spec.cols or proj.shape[1] != 2 * spec.cols or \
            any(v.dtype != torch.float32 or v.numel() != spec.cols for v in (rb, ib, decay)) or u.dtype != proj.dtype or \
            slots.dtype != torch.int32 or slots.numel() != table.batch:
        raise ValueError(f"lru_scan: shapes {tuple(z.shape)}, {tuple(proj.shape)} do not fit {spec}")
    out = torch.empty_like(u)
    a, t = spec.c(_dtype_code(proj)), table.c()
    check_layers(_lib.load_layers().ktk_lru_scan(
        _ptr(z), _ptr(u), _ptr(proj), proj.shape[1], 0, _ptr(new_indptr), rows, max_new, _ptr(slots), state.shape[0],
        _ptr(rb), _ptr(ib), _ptr(decay), _ptr(state), _ptr(out), ctypes.byref(t), ctypes.byref(a), _ptr(status), _stream()))
    _launched()
    return out


def lru_decode_supported(spec: LruSpec, dtype) -> bool:
    a = spec.c(_lib.KTK_BF16 if dtype == torch.bfloat16 else _lib.KTK_F32)
    return bool(_lib.load_layers().ktk_lru_decode_supported(ctypes.byref(a)))


def lru_decode(proj, spec: LruSpec, table: PageTable, slots, conv_w, conv_b, gates, rb, ib, decay, ring, state, status=None):
    """lru_conv, lru_gate_products and lru_scan of one token of every sequence, in one launch (bf16)."""
    _cuda(proj, slots, conv_w, conv_b, gates, rb, ib, decay, ring, state, status)
    n = pad8(spec.block)
    if proj.shape != (table.batch, 2 * spec.cols) or tuple(ring.shape[1:]) != (spec.taps, spec.cols) or \
            tuple(gates.shape) != (spec.blocks, 2 * n, n) or tuple(conv_w.shape) != (spec.taps, spec.cols) or \
            any(v.dtype != torch.float32 or v.numel() != spec.cols for v in (conv_b, rb, ib, decay)) or \
            any(v.dtype != torch.bfloat16 for v in (proj, ring, gates)) or conv_w.dtype != torch.float32 or \
            state.dtype != torch.float32 or state.shape != (ring.shape[0], spec.cols) or \
            slots.dtype != torch.int32 or slots.numel() != table.batch:
        raise ValueError(f"lru_decode: shapes {tuple(proj.shape)}, {tuple(ring.shape)} do not fit {spec}")
    out = torch.empty(proj.shape[0], spec.cols, dtype=proj.dtype, device=proj.device)
    a, t = spec.c(_lib.KTK_BF16), table.c()
    check_layers(_lib.load_layers().ktk_lru_decode(
        _ptr(proj), proj.shape[1], 0, spec.cols, proj.shape[0], _ptr(slots), ring.shape[0], _ptr(conv_w), _ptr(conv_b),
        _ptr(gates), _ptr(rb), _ptr(ib), _ptr(decay), _ptr(ring), _ptr(state), _ptr(out), ctypes.byref(t), ctypes.byref(a),
        _ptr(status), _stream()))
    _launched()
    return out
