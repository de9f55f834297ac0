"""Munadra: a decoder-only language model of latent-attention and gated linear-recurrence layers, with dense or
mixture-of-experts feed-forwards.

Only the sublayers' outputs are normalised (RMS norms with weights stored around zero); the sublayers read the fp32
residual stream itself:

    x <- x + norm1(mixer(x));    x <- x + norm2(feed_forward(x))      (the second part is optional)

* latent attention: per token one normalised latent and one rotated key part are cached; every head expands its keys and
  values from the latent.  Rotation of part of each head (YaRN stretch), a learned sink per head in the softmax, a
  sigmoid gate on every head's output.  A layer may read another layer's cache rows instead of writing its own.
* recurrence: a gated branch beside a causal convolution and a per-channel linear recurrence with real gates.
* experts: clamped gated activations, weights = the chosen experts' share of the softmax over all.
* the embedding is scaled, the logits (products with the embedding table) are scaled and soft-capped.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch
import torch.nn.functional as F

from . import layer_ops
from .layer_cache import LatentWeights, LruWeights
from .layer_ops import GateSpec, LatentSpec, LruSpec, MoeSpec, Rotation, pad8
from .layered_model import LayeredModel, WeightPacker

LRU_DECAY = 8.0                    # log a = -LRU_DECAY r softplus(lam)
EXPERT_SLOPE, EXPERT_SHIFT = 1.702, 1.0


@dataclass(frozen=True)
class MunadraLayer:
    """One layer: its mixer's spec and its feed-forward (`ff` > 0 and experts = 0: dense; ff = 0: none)."""
    mixer: Union[LatentSpec, LruSpec]
    ff: int = 0
    experts: int = 0
    top: int = 0
    limit: float = math.inf

    def moe(self, width: int) -> Optional[MoeSpec]:
        if not self.experts:
            return None
        return MoeSpec(self.experts, self.top, width, self.ff, score_all=True,
                       gate=GateSpec(self.limit, EXPERT_SLOPE, EXPERT_SHIFT))


@dataclass(frozen=True)
class MunadraConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float
    logit_scale: float
    logit_softcap: float
    layers: Tuple[MunadraLayer, ...]


def _rotation(rot: dict, dims: int, at: int) -> Rotation:
    if rot.get("dims", dims) != dims or dims % 2:
        raise ValueError(f"layer {at}: rotation of {rot.get('dims')} of {dims} rotated dimensions")
    s = rot.get("scaling")
    extra = {} if not s else dict(factor=s["factor"], original=s["original"], fast=s["fast"], slow=s["slow"], scaled=True)
    return Rotation(dims=dims, base=float(rot["base"]), **extra)


def _mixer_from(entry: dict, at: int, eps: float, before) -> Union[LatentSpec, LruSpec]:
    mx = entry["mixer"]
    if entry["type"] == "rglru":
        if mx["width"] % mx["blocks"]:
            raise ValueError(f"layer {at}: {mx['width']} channels in {mx['blocks']} blocks")
        return LruSpec(blocks=mx["blocks"], block=mx["width"] // mx["blocks"], taps=mx["conv"])
    if entry["type"] != "latent_attention":
        raise ValueError(f"layer {at}: mixer {entry['type']!r} (Munadra has 'latent_attention' and 'rglru')")
    spec = LatentSpec(heads=mx["heads"], dim=mx["dim"], rot_dim=mx["rot_dim"], vdim=mx["vdim"], rank=mx["kv_rank"],
                      scale=mx["scale"], rotation=_rotation(mx["rot"], mx["rot_dim"], at), eps=eps,
                      kv_from=mx.get("kv_from"))
    if spec.kv_from is not None:
        source = before[spec.kv_from].mixer if 0 <= spec.kv_from < at else None
        if not isinstance(source, LatentSpec) or source.kv_from is not None or \
                (source.rank, source.rot_dim, source.rotation) != (spec.rank, spec.rot_dim, spec.rotation):
            raise ValueError(f"layer {at}: kv_from {spec.kv_from} is no earlier latent layer with a cache of this shape")
    return spec


def _layer_from(entry: dict, at: int, eps: float, before) -> MunadraLayer:
    mixer, mlp = _mixer_from(entry, at, eps, before), entry.get("mlp")
    if mlp is None:
        return MunadraLayer(mixer)
    if mlp["kind"] == "dense":
        return MunadraLayer(mixer, ff=mlp["ff"])
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {at}: feed-forward {mlp['kind']!r} (Munadra has 'dense' and 'moe')")
    experts, top = mlp["router"]["experts"], mlp["router"]["top"]
    if not 0 < top <= experts:
        raise ValueError(f"layer {at}: {top} of {experts} experts")
    return MunadraLayer(mixer, ff=mlp["expert"]["ff"], experts=experts, top=top, limit=mlp["expert"]["limit"])


class Munadra(LayeredModel):
    @staticmethod
    def from_config(raw: dict) -> MunadraConfig:
        eps, layers = raw["norm"]["eps"], []
        for i, entry in enumerate(raw["layers"]):
            layers.append(_layer_from(entry, i, eps, layers))
        return MunadraConfig(vocab=raw["vocab"], width=raw["width"], norm_eps=eps,
                             embed_scale=raw["embedding"]["scale"], logit_scale=raw["logit_scale"],
                             logit_softcap=raw.get("logit_softcap") or 0.0, layers=tuple(layers))

    def __init__(self, config: MunadraConfig, weights, device, dtype=torch.bfloat16):
        """weights: mapping of the checkpoint's tensor names (``checkpoint.Checkpoint``, or a dict)."""
        super().__init__(config, device, dtype)
        pack, C = WeightPacker(weights, self.device, dtype), self.width

        def norm(name):                                  # weights around zero; no bias
            w = pack.vector(name, 1, C)
            w[:C] += 1.0
            return w, None
        self._load_table(pack)
        self.final_norm = norm("final.norm")
        for i, l in enumerate(config.layers):
            p = f"l{i}."
            layer = dict(norm1=norm(p + "norm1"), moe=l.moe(C))
            mixer = self._latent if isinstance(l.mixer, LatentSpec) else self._lru
            layer.update(mixer(pack, p + "mix.", l.mixer))
            if l.ff:
                layer.update(norm2=norm(p + "norm2"))
            elif p + "norm2" in weights:                 # nothing to normalise
                pack[p + "norm2"]
            if l.experts:
                layer.update(pack.experts(p + "mlp.", layer["moe"], bias=False))
            elif l.ff:
                layer.update(dense=torch.cat((pack.matrix(p + "mlp.gate", l.ff, C), pack.matrix(p + "mlp.up", l.ff, C))),
                             dense_down=pack.matrix(p + "mlp.down", C, l.ff))
            self.layers.append(layer)
            self.cache_specs.append(l.mixer)

    def _latent(self, pack, mx, s: LatentSpec) -> dict:
        C, own = self.width, s.kv_from is None
        q = pack[mx + "q"]
        if tuple(q.shape) != (s.heads * (s.dim + s.rot_dim), C):
            raise ValueError(f"{mx}q: shape {tuple(q.shape)}, expected {(s.heads * (s.dim + s.rot_dim), C)}")
        rows = pack.zeros(s.heads, s.head_cols, pad8(C))          # heads of [dim | rotated], each part padded
        q = q.view(s.heads, s.dim + s.rot_dim, C)
        rows[:, :s.dim, :C] = q[:, :s.dim]
        rows[:, pad8(s.dim):pad8(s.dim) + s.rot_dim, :C] = q[:, s.dim:]
        parts = [rows.view(-1, pad8(C))]
        if own:
            kv = pack[mx + "dkv"]
            if tuple(kv.shape) != (s.rank + s.rot_dim, C):
                raise ValueError(f"{mx}dkv: shape {tuple(kv.shape)}, expected {(s.rank + s.rot_dim, C)}")
            rows = pack.zeros(s.row_cols, pad8(C))
            rows[:s.rank, :C] = kv[:s.rank]
            rows[pad8(s.rank):pad8(s.rank) + s.rot_dim, :C] = kv[s.rank:]
            parts.append(rows)
        parts.append(pack.matrix(mx + "g", s.heads, C))
        ukv = torch.cat((pack.matrix(mx + "uk", (s.heads, s.dim), s.rank), pack.matrix(mx + "uv", (s.heads, s.vdim), s.rank)))
        cut = s.heads * pad8(s.dim)
        sink = pack.vector(mx + "sink", 1, s.heads)[:s.heads].contiguous()
        w = LatentWeights(ukv=ukv, uk=ukv[:cut].view(s.heads, -1, pad8(s.rank)), uv=ukv[cut:].view(s.heads, -1, pad8(s.rank)),
                          sink=sink, norm=pack.vector(mx + "dkv.norm", 1, s.rank) if own else None,
                          turns=s.rotation.turns().to(self.device))
        return dict(proj=torch.cat(parts), proj_b=None, out=pack.matrix(mx + "o", C, (s.heads, s.vdim)), mix=w)

    def _lru(self, pack, mx, s: LruSpec) -> dict:
        C, n, bs = self.width, s.blocks * s.block, pad8(s.block)
        spread = (s.blocks, s.block)
        vector = lambda name, to=torch.float32: pack.vector(mx + name, s.blocks, s.block, to)
        gates = pack.zeros(s.blocks, 2, bs, bs)
        for k, name in enumerate(("ra", "ri")):
            t = pack[mx + name]
            if tuple(t.shape) != (s.blocks, s.block, s.block):
                raise ValueError(f"{mx}{name}: shape {tuple(t.shape)}, expected {(s.blocks, s.block, s.block)}")
            gates[:, k, :s.block, :s.block] = t
        t = pack[mx + "conv"]
        if tuple(t.shape) != (n, s.taps):
            raise ValueError(f"{mx}conv: shape {tuple(t.shape)}, expected {(n, s.taps)}")
        conv = pack.zeros(s.taps, s.blocks, bs, dtype=torch.float32)
        conv[:, :, :s.block] = t.t().reshape(s.taps, s.blocks, s.block).float()
        lam = pack.vector(mx + "lam", s.blocks, s.block, torch.float64)
        w = LruWeights(conv_w=conv.view(s.taps, -1), conv_b=vector("conv.b"), gates=gates.view(s.blocks, 2 * bs, bs),
                       rb=vector("ra.b"), ib=vector("ri.b"), decay=(LRU_DECAY * F.softplus(lam)).float())
        return dict(proj=torch.cat((pack.matrix(mx + "y", spread, C), pack.matrix(mx + "x", spread, C))),
                    proj_b=torch.cat((vector("y.b", self.dtype), vector("x.b", self.dtype))),
                    out=pack.matrix(mx + "o", C, spread), mix=w)

    # ---- forward
    def _hidden(self, input_ids, batch_idx, kv, streams=None):
        """The final norm of every row, [rows, stride].  `streams`, a list, receives the residual stream behind every
        layer (a debugging aid)."""
        x, h, step = self._stream(input_ids, center=False)
        seq_len = input_ids.shape[1]
        step(tokens=input_ids.reshape(-1).to(torch.int64).contiguous(), embed=self.embed, embed_scale=self.config.embed_scale,
             pre=None if self.layers else self.final_norm)
        for i, L in enumerate(self.layers):
            after = None if i + 1 < len(self.layers) else self.final_norm     # a sublayer reads the stream as it is
            last = L["norm2"] if "norm2" in L else None
            proj = torch.mm(h, L["proj"].t()) if L["proj_b"] is None else torch.addmm(L["proj_b"], h, L["proj"].t())
            mix = kv.attend_latent if isinstance(L["mix"], LatentWeights) else kv.recur
            y = torch.mm(mix(proj, i, batch_idx, seq_len, L["mix"]), L["out"].t())
            step(y=y, post=L["norm1"], pre=None if last else after, zero=L.get("counts"))
            if L["moe"] is not None:
                step(y=self._experts(h, L), parts=L["moe"].top, post=last, pre=after)
            elif last:
                inner = layer_ops.gated_rows(torch.mm(h, L["dense"].t()))
                step(y=torch.mm(inner, L["dense_down"].t()), post=last, pre=after)
            if streams is not None:
                streams.append(x[:, :self.width].clone())
        return h

    def _logits(self, h):
        return layer_ops.scale_cap(self._project(h), self.config.logit_scale, self.config.logit_softcap)

    def _best(self, h):
        if self.config.logit_scale > 0:                  # scale and softcap keep the order
            return self._project(h).argmax(dim=-1)
        return self._logits(h).argmax(dim=-1)


def random_weights(config: MunadraConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> dict:
    """Random tensors under the checkpoint's names (tests and benchmarks): projections with variance 1 / fan-in, norm
    weights around zero, decays spread over short and long memories."""
    g = torch.Generator(device=device).manual_seed(seed)
    C, W = config.width, {}

    def put(name, *shape, std=None, mean=0.0):
        std = 1.0 / math.sqrt(shape[-1]) if std is None else std
        W[name] = (torch.randn(*shape, generator=g, device=device) * std + mean).to(dtype)

    put("embed", config.vocab, C, std=1.0)
    for i, l in enumerate(config.layers):
        p, mx, s = f"l{i}.", f"l{i}.mix.", l.mixer
        for n in ("norm1",) + (("norm2",) if l.ff else ()):
            put(p + n, C, std=0.1)
        if isinstance(s, LatentSpec):
            put(mx + "q", s.heads * (s.dim + s.rot_dim), C)
            if s.kv_from is None:
                put(mx + "dkv", s.rank + s.rot_dim, C)
                put(mx + "dkv.norm", s.rank, std=0.1, mean=1.0)
            put(mx + "uk", s.heads * s.dim, s.rank)
            put(mx + "uv", s.heads * s.vdim, s.rank)
            put(mx + "sink", s.heads, std=1.0)
            put(mx + "g", s.heads, C)
            put(mx + "o", C, s.heads * s.vdim)
        else:
            n = s.blocks * s.block
            for b in ("y", "x"):
                put(mx + b, n, C)
                put(f"{mx}{b}.b", n, std=0.1)
            put(mx + "conv", n, s.taps)
            put(mx + "conv.b", n, std=0.1)
            for r in ("ra", "ri"):
                put(mx + r, s.blocks, s.block, s.block)
                put(f"{mx}{r}.b", s.blocks, s.block, std=0.5)
            put(mx + "lam", n, std=1.5, mean=-4.0)
            put(mx + "o", C, n)
        if l.experts:
            for e in range(l.experts):
                put(f"{p}mlp.e{e}.gate", l.ff, C)
                put(f"{p}mlp.e{e}.up", l.ff, C)
                put(f"{p}mlp.e{e}.down", C, l.ff)
            put(p + "mlp.router", l.experts, C)
        elif l.ff:
            put(p + "mlp.gate", l.ff, C)
            put(p + "mlp.up", l.ff, C)
            put(p + "mlp.down", C, l.ff)
    put("final.norm", C, std=0.1)
    return W
