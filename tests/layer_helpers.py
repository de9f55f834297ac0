"""Builders for the layer-mechanism tests: small random Gifetar models, paged caches with free head sizes, inputs in
which single keys stand out."""
from __future__ import annotations

import torch

from oracle import gifetar as plain


def small_config(layers=None, vocab=101, width=72, eps=1e-5, mult=0.4):
    """A config.json dict whose layers differ from one another in every size and constant."""
    if layers is None:
        layers = [
            layer_entry(4, 2, 24, 40, experts=5, top=2, ff=56, diff=0.2, softcap=12.0, coef=0.4, every=16),
            layer_entry(3, 1, 16, 16, experts=0, diff=0.5, softcap=80.0, coef=0.1, every=7),
            layer_entry(2, 2, 64, 72, experts=3, top=3, ff=24, diff=0.35, softcap=30.0, coef=0.7, every=50),
            layer_entry(8, 1, 40, 96, experts=7, top=1, ff=40, diff=0.1, softcap=45.0, coef=0.3, every=33),
        ]
    return {"architecture": "Gifetar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": layers}


def layer_entry(heads, kv_heads, dim, vdim, experts, top=0, ff=0, diff=0.3, softcap=30.0, coef=0.5, every=64,
                scale=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "softcap": softcap,
             "scale": scale if scale is not None else 1.3 * dim ** -0.5, "q_temp": {"coef": coef, "every": every}}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}} if experts else None
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def random_model(raw, seed=0, boost=2.0):
    """Random bf16 weights for a config dict.  boost: factor on the query projections, so that attention is peaked and
    a wrong key shows."""
    from kinetics_b200.gifetar import Gifetar, random_weights
    W = random_weights(Gifetar.from_config(raw), seed)
    for name in W:
        if name.endswith("mix.q"):
            W[name] = (W[name].float() * boost).to(torch.bfloat16)
    return W


def clear_routes(W, seed=0):
    """The same weights with routers whose choice is clear at every token (far apart biases): in bf16 no decision then
    hangs on a rounding."""
    g = torch.Generator().manual_seed(seed)
    W = dict(W)
    for name in W:
        if name.endswith("mlp.router"):
            n = W[name].shape[0]
            W[name] = (W[name].float() * 0.05).to(torch.bfloat16)
            W[name + ".b"] = torch.linspace(-0.5 * n, 0.5 * n, n)[torch.randperm(n, generator=g)].to(torch.bfloat16)
    return W


def as_dtype(W, dtype):
    return {k: v.to(dtype) for k, v in W.items()}


def standout_inputs(total, first, heads, kv_heads, dim, vdim, edges, seed=0, strength=5.0, maps=2):
    """q [total - first, heads, maps, dim], k [total, kv_heads, maps, dim], v [total, kv_heads, vdim]: keys at the
    `edges` positions are long vectors of their own direction; each query row points along one of them (its own
    position's and the next one's neighbours included), so that score stands out wherever the key is visible."""
    g = torch.Generator().manual_seed(seed)
    rows = total - first
    k = 0.3 * torch.randn(total, kv_heads, maps, dim, generator=g)
    v = torch.randn(total, kv_heads, vdim, generator=g)
    unit = lambda *s: torch.nn.functional.normalize(torch.randn(*s, generator=g), dim=-1)
    q = 0.3 * torch.randn(rows, heads, maps, dim, generator=g)
    edges = [e for e in sorted(set(edges)) if 0 <= e < total]
    dirs = unit(len(edges), kv_heads, maps, dim)
    for n, e in enumerate(edges):
        k[e] = strength * dirs[n]
    pick = torch.randint(0, len(edges), (rows, heads, maps), generator=g)
    group = heads // kv_heads
    for h in range(heads):
        for m in range(maps):
            q[:, h, m] += strength * dirs[pick[:, h, m], h // group, m]
    return q, k, v


class PagedCase:
    """Contiguous keys and values of several sequences in a permuted paged cache; unused slots hold NaN."""

    def __init__(self, ks, vs, dtype, page_size, device, seed=0, dim_stride=None, vdim_stride=None):
        from kinetics_b200.layer_ops import PageTable, pad8
        g = torch.Generator().manual_seed(seed)
        ps = page_size
        lens = [k.shape[0] for k in ks]
        pages = [(n + ps - 1) // ps for n in lens]
        total = sum(pages) + 3
        perm = torch.randperm(total, generator=g).tolist()
        Gm, d = ks[0].shape[1] * ks[0].shape[2], ks[0].shape[3]
        G, dv = vs[0].shape[1], vs[0].shape[2]
        K = torch.full((total * ps, Gm, pad8(d)), float("nan"))
        V = torch.full((total * ps, G, pad8(dv)), float("nan"))
        idx, indptr, last = [], [0], []
        for k, v, n, c in zip(ks, vs, lens, pages):
            mine = [perm.pop() for _ in range(c)]
            idx += mine
            indptr.append(len(idx))
            last.append(n - (c - 1) * ps if c else 0)
            slots = torch.tensor([mine[t // ps] * ps + t % ps for t in range(n)], dtype=torch.long)
            if n:
                K[slots] = torch.nn.functional.pad(k.reshape(n, Gm, d), (0, pad8(d) - d))
                V[slots] = torch.nn.functional.pad(v, (0, pad8(dv) - dv))
        pages_of = lambda t, heads, cols: t.view(total, ps, heads, cols).transpose(1, 2).contiguous().to(dtype).to(device)
        self.k, self.v = pages_of(K, Gm, pad8(d)), pages_of(V, G, pad8(dv))
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
        self.table = PageTable(i32(idx or [0]), i32(indptr), i32(last), ps, total)


def pad_q(q, device, dtype):
    """[rows, heads, maps, dim] -> the projection rows the kernels read."""
    from kinetics_b200.layer_ops import pad8
    rows, _, _, d = q.shape
    return torch.nn.functional.pad(q, (0, pad8(d) - d)).reshape(rows, -1).to(dtype).to(device).contiguous()


def plain_attention(q, k, v, spec, first):
    mixer = {"q_temp": {"coef": spec.temp_coef, "every": spec.temp_every}, "scale": spec.scale,
             "softcap": spec.softcap if spec.softcap > 0 else 1e30, "diff": 1.0 - spec.out_scale}
    return plain.difference_attention(q.double(), k.double(), v.double(), mixer, spec.lam, spec.eps, first)


def rms(x):
    return float(x.double().pow(2).mean().sqrt())
