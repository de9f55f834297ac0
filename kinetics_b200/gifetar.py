"""Gifetar: a decoder-only language model of differential attention and mixture-of-experts layers.

Every sublayer is normalised on both sides (layer norms with bias) and enters the fp32 residual stream with a fixed
multiplier m:

    x <- x + m norm1b(attention(norm1(x)));    x <- x + m norm2b(experts(norm2(x)))      (the second part is optional)

* attention: per head two softmax maps over the same values, a1 - lambda a2, unit RMS norm over the head, times
  (1 - diff); scores are scaled, multiplied with the query's temperature (which grows with the position) and
  soft-capped; no rotation, biases in the q, k and v projections.
* experts: each token uses the best `top` of the layer's gated feed-forwards, weighted by the softmax over the chosen
  router logits.
* the logits are the final norm's output times the embedding table.

A decode layer is: qkv GEMM, append, attention, output GEMM, one row kernel (post-norm, residual, next norm), router,
two expert GEMMs, and the same row kernel over the experts' parts.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from .layer_ops import AttentionSpec, MoeSpec
from .layered_model import LayeredModel, WeightPacker


@dataclass(frozen=True)
class GifetarLayer:
    """One layer's sizes and constants; `experts` = 0: no feed-forward."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    diff: float
    temp_coef: float
    temp_every: float
    experts: int = 0
    top: int = 0
    ff: int = 0

    def attention(self, lam: float, eps: float) -> AttentionSpec:
        return AttentionSpec(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale,
                             maps=2, softcap=self.softcap, temp_coef=self.temp_coef, temp_every=self.temp_every,
                             lam=lam, eps=eps, out_scale=1.0 - self.diff)

    def moe(self, width: int) -> Optional[MoeSpec]:
        return MoeSpec(self.experts, self.top, width, self.ff) if self.experts else None


@dataclass(frozen=True)
class GifetarConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[GifetarLayer, ...]


def _layer_from(entry: dict, at: int) -> GifetarLayer:
    if entry["type"] != "attention":
        raise ValueError(f"layer {at}: mixer {entry['type']!r} (Gifetar has 'attention')")
    mx, mlp = entry["mixer"], entry.get("mlp")
    if mx["heads"] % mx["kv_heads"]:
        raise ValueError(f"layer {at}: {mx['heads']} heads over {mx['kv_heads']} key/value heads")
    temp = mx.get("q_temp") or {"coef": 0.0, "every": 1.0}
    extra = {}
    if mlp is not None:
        if mlp.get("kind", "moe") != "moe":
            raise ValueError(f"layer {at}: feed-forward {mlp['kind']!r} (Gifetar has 'moe')")
        extra = dict(experts=mlp["router"]["experts"], top=mlp["router"]["top"], ff=mlp["expert"]["ff"])
        if not 0 < extra["top"] <= extra["experts"]:
            raise ValueError(f"layer {at}: {extra['top']} of {extra['experts']} experts")
    return GifetarLayer(heads=mx["heads"], kv_heads=mx["kv_heads"], dim=mx["dim"], vdim=mx["vdim"],
                        scale=mx["scale"], softcap=mx.get("softcap") or 0.0, diff=mx["diff"], temp_coef=temp["coef"],
                        temp_every=temp["every"], **extra)


class Gifetar(LayeredModel):
    @staticmethod
    def from_config(raw: dict) -> GifetarConfig:
        return GifetarConfig(vocab=raw["vocab"], width=raw["width"], norm_eps=raw["norm"]["eps"],
                             residual_mult=raw["residual_mult"],
                             layers=tuple(_layer_from(e, i) for i, e in enumerate(raw["layers"])))

    def __init__(self, config: GifetarConfig, weights, device, dtype=torch.bfloat16):
        """weights: mapping of the checkpoint's tensor names (``checkpoint.Checkpoint``, or a dict)."""
        super().__init__(config, device, dtype)
        pack, C = WeightPacker(weights, self.device, dtype), self.width
        self.mult = config.residual_mult
        norm = lambda name: (pack.vector(name, 1, C), pack.vector(name + ".b", 1, C))
        self._load_table(pack)
        self.final_norm = norm("final.norm")
        for i, l in enumerate(config.layers):
            p, mx = f"l{i}.", f"l{i}.mix."
            H2, G2 = l.heads * 2, l.kv_heads * 2
            dot = lambda a, b: float((pack[mx + a].double() * pack[mx + b].double()).sum())
            lam = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + l.diff
            spec = l.attention(lam, self.eps)
            layer = dict(
                norm1=norm(p + "norm1"), norm1b=norm(p + "norm1b"), spec=spec, moe=l.moe(C),
                wqkv=torch.cat((pack.matrix(mx + "q", (H2, l.dim), C), pack.matrix(mx + "k", (G2, l.dim), C),
                                pack.matrix(mx + "v", (l.kv_heads, l.vdim), C))),
                bqkv=torch.cat((pack.vector(mx + "q.b", H2, l.dim, dtype), pack.vector(mx + "k.b", G2, l.dim, dtype),
                                pack.vector(mx + "v.b", l.kv_heads, l.vdim, dtype))),
                wo=pack.matrix(mx + "o", C, (l.heads, l.vdim)))
            if layer["moe"] is not None:
                layer.update(norm2=norm(p + "norm2"), norm2b=norm(p + "norm2b"),
                             **pack.experts(p + "mlp.", layer["moe"], bias=True))
            self.layers.append(layer)
            self.cache_specs.append(spec)

    def _hidden(self, input_ids, batch_idx, kv, streams=None):
        """The final norm of every row, [rows, stride].  `streams`, a list, receives the residual stream behind every
        layer (a debugging aid)."""
        x, h, step = self._stream(input_ids)
        step(tokens=input_ids.reshape(-1).to(torch.int64).contiguous(), embed=self.embed,
             pre=self.layers[0]["norm1"] if self.layers else self.final_norm)
        for i, L in enumerate(self.layers):
            after = self.layers[i + 1]["norm1"] if i + 1 < len(self.layers) else self.final_norm
            proj = torch.addmm(L["bqkv"], h, L["wqkv"].t())
            attn = kv.attend(proj, i, batch_idx, input_ids.shape[1])
            y = torch.mm(attn, L["wo"].t())
            if L["moe"] is None:
                step(y=y, post=L["norm1b"], mult=self.mult, pre=after)
            else:
                step(y=y, post=L["norm1b"], mult=self.mult, pre=L["norm2"], zero=L["counts"])
                step(y=self._experts(h, L), parts=L["moe"].top, post=L["norm2b"], mult=self.mult, pre=after)
            if streams is not None:
                streams.append(x[:, :self.width].clone())
        return h


def random_weights(config: GifetarConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> dict:
    """Random tensors under the checkpoint's names (tests and benchmarks): projections with variance 1 / fan-in, norm
    weights around 1."""
    g = torch.Generator(device=device).manual_seed(seed)
    C, W = config.width, {}

    def put(name, *shape, std=None, mean=0.0):
        std = 1.0 / math.sqrt(shape[-1]) if std is None else std
        W[name] = (torch.randn(*shape, generator=g, device=device) * std + mean).to(dtype)

    def norm(name):
        put(name, C, std=0.1, mean=1.0)
        put(name + ".b", C, std=0.1)

    put("embed", config.vocab, C, std=1.0)
    for i, l in enumerate(config.layers):
        p, mx = f"l{i}.", f"l{i}.mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l.experts else ()):
            norm(p + n)
        for n, rows in (("q", l.heads * 2 * l.dim), ("k", l.kv_heads * 2 * l.dim), ("v", l.kv_heads * l.vdim)):
            put(mx + n, rows, C)
            put(f"{mx}{n}.b", rows, std=0.1)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            put(mx + n, l.dim, std=0.1)
        put(mx + "o", C, l.heads * l.vdim)
        for e in range(l.experts):
            put(f"{p}mlp.e{e}.gate", l.ff, C)
            put(f"{p}mlp.e{e}.up", l.ff, C)
            put(f"{p}mlp.e{e}.down", C, l.ff)
        if l.experts:
            put(p + "mlp.router", l.experts, C)
            put(p + "mlp.router.b", l.experts, std=0.1)
    norm("final.norm")
    return W
