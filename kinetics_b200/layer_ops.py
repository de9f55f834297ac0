"""Wrappers of libktk_layers.so (``include/ktk_layers.h``): layer mechanisms whose sizes and constants are parameters.

Every call runs a hand-written CUDA kernel on the current stream; a CPU tensor raises.  ``variant`` picks a kernel
(``VARIANT_AUTO``: the fastest built one for the sizes); the fp32 forms and odd sizes run on the FMA kernels.
"""
from __future__ import annotations

import ctypes
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
    softcap tanh(score / softcap) if softcap > 0."""
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
                         self.out_scale)


@dataclass(frozen=True)
class MoeSpec:
    """A mixture of experts: each row uses the `top` of `experts` gated feed-forwards of inner size ff."""
    experts: int
    top: int
    width: int
    ff: int

    def c(self, dtype_code: int) -> _lib.Moe:
        return _lib.Moe(self.experts, self.top, self.width, self.ff, pad8(self.width), pad8(self.ff), dtype_code, 0)


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
                  tokens=None, embed=None, center: bool = True, zero=None, status=None) -> None:
    """Rows of the fp32 residual stream x [rows, stride], in place: x = embed[tokens] (if given); x += mult *
    norm(sum of y [rows, parts, stride]; post) (if y is given; post None: no norm); h = norm(x; pre) in the dtype
    of h (if h is given).  pre / post: (weight, bias or None), fp32 [stride].  zero: an int32 tensor to clear."""
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
        _ptr(tokens), _ptr(embed), 0 if embed is None else embed.shape[0], _ptr(x), _ptr(y), parts, _ptr(pw), _ptr(pb),
        mult, _ptr(nw), _ptr(nb), _ptr(h), eps, int(center), rows, cols, stride, _ptr(zero),
        0 if zero is None else zero.numel(), code, _ptr(status), _stream()))
    _launched()


def _cache_check(spec: AttentionSpec, table: PageTable, k_pages, v_pages):
    if tuple(k_pages.shape) != (table.num_pages, spec.kv_heads * spec.maps, table.page_size, spec.dim_stride) or \
            tuple(v_pages.shape) != (table.num_pages, spec.kv_heads, table.page_size, spec.vdim_stride):
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


def attention_splits(spec: AttentionSpec, batch: int, max_keys: int, dtype) -> int:
    a = spec.c(_lib.KTK_BF16 if dtype == torch.bfloat16 else _lib.KTK_F32)
    return int(_lib.load_layers().ktk_paged_attention_splits(ctypes.byref(a), batch, max_keys))


def attention_workspace(spec: AttentionSpec, rows: int, splits: int, dtype) -> int:
    a = spec.c(_lib.KTK_BF16 if dtype == torch.bfloat16 else _lib.KTK_F32)
    return int(_lib.load_layers().ktk_paged_attention_workspace(ctypes.byref(a), rows, splits))


def paged_attention(proj, k_pages, v_pages, table: PageTable, spec: AttentionSpec, new_indptr=None, max_new: int = 1,
                    splits: int = 1, workspace=None, variant: int = VARIANT_AUTO, out=None, status=None):
    """Causal attention of the rows of proj (whose first spec.q_cols columns are the queries) over their sequences;
    their keys are already in the pages.  new_indptr int32 [batch + 1]: rows per sequence; None: one each.
    Returns [rows, heads * vdim_stride]."""
    _cuda(proj, k_pages, v_pages, new_indptr, workspace, out, status)
    _cache_check(spec, table, k_pages, v_pages)
    if proj.dtype != k_pages.dtype or v_pages.dtype != k_pages.dtype:
        raise TypeError("paged_attention: proj and the cache share a dtype")
    a, t = spec.c(_dtype_code(k_pages)), table.c()
    rows = proj.shape[0]
    if out is None:
        out = torch.empty(rows, spec.o_cols, dtype=proj.dtype, device=proj.device)
    if new_indptr is None and workspace is None:
        need = attention_workspace(spec, rows, splits, proj.dtype)
        if need:
            workspace = torch.empty(need, dtype=torch.uint8, device=proj.device)
    wsb = 0 if workspace is None else workspace.numel()
    check_layers(_lib.load_layers().ktk_paged_attention(
        _ptr(proj), proj.shape[1], _ptr(new_indptr), rows, max_new, _ptr(k_pages), _ptr(v_pages), ctypes.byref(t),
        _ptr(out), _ptr(workspace), wsb, splits, variant, ctypes.byref(a), _ptr(status), _stream()))
    _launched(2 if new_indptr is None and splits > 1 else 1)
    return out


class Routing:
    """Where the rows of a step go: ids / weights [rows, top], counts [experts], bucket [experts, rows]."""

    def __init__(self, spec: MoeSpec, rows: int, device, counts: Optional[torch.Tensor] = None):
        self.ids = torch.empty(rows, spec.top, dtype=torch.int32, device=device)
        self.weights = torch.empty(rows, spec.top, dtype=torch.float32, device=device)
        self.counts = counts if counts is not None else torch.zeros(spec.experts, dtype=torch.int32, device=device)
        self.bucket = torch.empty(spec.experts, rows, dtype=torch.int32, device=device)


def moe_route(h, w, b, spec: MoeSpec, counts=None, variant: int = VARIANT_AUTO) -> Routing:
    """Router of rows h [rows, pad8(width)]: w [experts, pad8(width)] in the dtype of h, b fp32 [experts].  counts:
    a cleared int32 [experts] tensor to count into (None: a new one)."""
    _cuda(h, w, b, counts)
    if w.dtype != h.dtype or b.dtype != torch.float32 or tuple(w.shape) != (spec.experts, h.shape[1]):
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
