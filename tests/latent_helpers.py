"""Builders for the tests of latent attention and the linear recurrence: small random Munadra models, cached rows in
permuted pages, queries that single out one far key."""
from __future__ import annotations

import torch

from oracle import munadra as plain


def rot(dims, base=10000.0, factor=None, original=64, fast=8.0, slow=0.5):
    out = {"base": base, "dims": dims}
    if factor is not None:
        out["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return out


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def latent(heads, dim, rot_dim, vdim, rank, mlp, scale=None, kv_from=None, **rotation):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": rot(rot_dim, **rotation),
             "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def rglru(width, blocks, conv, mlp):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def small_config(layers=None, vocab=93, width=72, eps=1e-5, embed_scale=1.7, logit_scale=0.3, softcap=9.0):
    """A config.json dict whose layers differ from one another in every size and constant."""
    if layers is None:
        layers = [
            latent(3, 24, 16, 40, 56, moe(5, 2, 40), factor=4.0),
            rglru(60, 3, 4, dense(88)),
            latent(2, 16, 8, 24, 48, None, base=500.0),
            latent(5, 40, 16, 16, 56, moe(3, 3, 24, limit=0.7), kv_from=0, factor=4.0),
            rglru(48, 1, 2, moe(7, 1, 56, limit=3.0)),
        ]
    return {"architecture": "Munadra", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "logit_scale": logit_scale, "logit_softcap": softcap, "layers": layers}


def random_model(raw, seed=0, boost=2.5):
    """Random bf16 weights for a config dict.  boost: factor on the query projections, so that attention is peaked and a
    wrong key shows."""
    from kinetics_b200.munadra import Munadra, random_weights
    W = random_weights(Munadra.from_config(raw), seed)
    for name in W:
        if name.endswith("mix.q"):
            W[name] = (W[name].float() * boost).to(torch.bfloat16)
    return W


def quiet_experts(W):
    """The same weights with small norms behind the mixtures of experts: in bf16, where a close choice of an expert hangs
    on rounding, it then moves the stream little."""
    W = dict(W)
    for name in W:
        if name.endswith("mlp.router"):
            norm = name.replace("mlp.router", "norm2")
            W[norm] = (0.08 * (1 + W[norm].float()) - 1).to(torch.bfloat16)
    return W


def as_dtype(W, dtype):
    return {k: v.to(dtype) for k, v in W.items()}


def rms(x):
    return float(x.double().pow(2).mean().sqrt())


# ---- rows that all heads share, in pages
class RowPages:
    """Contiguous rows [tokens, cols] of several sequences in permuted pages of a tensor full of NaN."""

    def __init__(self, rows, dtype, page_size, device, seed=0, extra=3):
        from kinetics_b200.layer_ops import PageTable
        g = torch.Generator().manual_seed(seed)
        lens = [r.shape[0] for r in rows]
        pages = [(n + page_size - 1) // page_size for n in lens]
        total = sum(pages) + extra
        perm = torch.randperm(total, generator=g).tolist()
        data = torch.full((total * page_size, rows[0].shape[1]), float("nan"))
        idx, indptr, last = [], [0], []
        self.slots = []
        for r, n, c in zip(rows, lens, pages):
            mine = [perm.pop() for _ in range(c)]
            idx += mine
            indptr.append(len(idx))
            last.append(n - (c - 1) * page_size if c else 0)
            self.slots.append(torch.tensor([mine[t // page_size] * page_size + t % page_size for t in range(n)]))
            data[self.slots[-1]] = r.float()
        self.pages = data.view(total, 1, page_size, -1).to(dtype).to(device)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
        self.table = PageTable(i32(idx or [0]), i32(indptr), i32(last), page_size, total)

    def row(self, sequence):
        """The rows of a sequence as they lie in the pages now."""
        flat = self.pages.view(-1, self.pages.shape[-1])
        return flat[self.slots[sequence].to(flat.device)]


def pointed_rows(total, first, heads, cols, edges, seed=0, strength=5.0):
    """q [total - first, heads, cols], k [total, cols]: keys at the `edges` are long vectors of their own direction and
    each query points along one of them, so its score stands out wherever the key is visible."""
    g = torch.Generator().manual_seed(seed)
    rows = total - first
    k = 0.3 * torch.randn(total, cols, generator=g)
    q = 0.3 * torch.randn(rows, heads, cols, generator=g)
    edges = [e for e in sorted(set(edges)) if 0 <= e < total]
    dirs = torch.nn.functional.normalize(torch.randn(len(edges), cols, generator=g), dim=-1)
    k[edges] = strength * dirs
    q += strength * dirs[torch.randint(0, len(edges), (rows, heads), generator=g)]
    return q, k


def plain_rows(q, k, vdim, scale, sink, gate, first):
    """Attention over shared rows, the first vdim columns being the values: q [rows, heads, cols] -> [rows, heads, vdim]."""
    out = []
    for h in range(q.shape[1]):
        p = plain.sink_softmax(q[:, h] @ k.t() * scale, sink[h], first)
        o = p @ k[:, :vdim]
        out.append(o if gate is None else plain.sigmoid(gate[:, h:h + 1]) * o)
    return torch.stack(out, dim=1)
