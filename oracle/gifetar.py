"""Plain restatement of the Gifetar language model on the CPU, for the tests.

One function per mechanism, written straight from its formula with full score matrices and per-token expert
loops; nothing is shared with the product's code.  Everything runs in the dtype of the weights it is given
(float32, or float64 for a sharper yardstick).

Weights are a dict name -> tensor with the checkpoint's names; `config` is the dict of a config.json.
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, b, eps):
    """x [..., n]: centred, divided by the root of (mean squared deviation + eps), times w, plus b."""
    d = x - x.mean(dim=-1, keepdim=True)
    var = (d * d).mean(dim=-1, keepdim=True)
    return d / torch.sqrt(var + eps) * w + b


def rms_unit(x, eps):
    """x [..., n] divided by sqrt(mean square + eps)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def query_temperature(positions, coef, every):
    """Factor of the query at each position: 1 + coef ln(floor((p + 1) / every) + 1)."""
    steps = torch.floor((positions.to(torch.float64) + 1.0) / every)
    return 1.0 + coef * torch.log(steps + 1.0)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def causal_softmax(scores, first):
    """scores [rows, keys]; row i stands at position first + i and sees the keys at positions <= its own."""
    rows, keys = scores.shape
    at = first + torch.arange(rows).unsqueeze(1)
    seen = torch.arange(keys).unsqueeze(0) <= at
    return torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)


def difference_attention(q, k, v, mixer, lam, eps, first=0):
    """q [rows, heads, 2, dim] at positions first.., k [keys, kv_heads, 2, dim], v [keys, kv_heads, vdim] ->
    [rows, heads, vdim]: two softmax maps per head over shared values, their weighted difference, unit norm."""
    rows, H = q.shape[:2]
    G = k.shape[1]
    q = q * query_temperature(first + torch.arange(rows), mixer["q_temp"]["coef"],
                              mixer["q_temp"]["every"]).to(q.dtype).view(-1, 1, 1, 1)
    out = torch.empty(rows, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        maps = []
        for m in range(2):
            s = soft_cap(q[:, h, m] @ k[:, g, m].t() * mixer["scale"], mixer["softcap"])
            maps.append(causal_softmax(s, first) @ v[:, g])
        out[:, h] = rms_unit(maps[0] - lam * maps[1], eps) * (1.0 - mixer["diff"])
    return out


def route(h, w, b, top):
    """h [rows, width] -> (expert ids [rows, top], weights [rows, top]): softmax over the chosen logits only."""
    z = h @ w.t() + b
    best, ids = torch.topk(z, top, dim=-1)
    return ids, torch.softmax(best, dim=-1)


def expert(h, gate, up, down):
    g = h @ gate.t()
    return (g * torch.sigmoid(g) * (h @ up.t())) @ down.t()


def mixture(h, W, prefix, mlp):
    """The mixture-of-experts feed-forward of one layer, row by row."""
    ids, weights = route(h, W[prefix + "router"], W[prefix + "router.b"], mlp["router"]["top"])
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            part = expert(h[rows], W[f"{prefix}e{e}.gate"], W[f"{prefix}e{e}.up"], W[f"{prefix}e{e}.down"])
            y[rows] += weights[rows, place].unsqueeze(1) * part
    return y


class History:
    """Keys and values of the tokens a sequence has run so far, per layer."""

    def __init__(self, layers):
        self.k, self.v = [None] * layers, [None] * layers

    def add(self, i, k, v):
        self.k[i] = k if self.k[i] is None else torch.cat((self.k[i], k))
        self.v[i] = v if self.v[i] is None else torch.cat((self.v[i], v))
        return self.k[i], self.v[i]


def attention_layer(h, W, prefix, mixer, eps, history, i):
    H, G, d, dv = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    rows = h.shape[0]
    q = (h @ W[prefix + "q"].t() + W[prefix + "q.b"]).view(rows, H, 2, d)
    k = (h @ W[prefix + "k"].t() + W[prefix + "k.b"]).view(rows, G, 2, d)
    v = (h @ W[prefix + "v"].t() + W[prefix + "v.b"]).view(rows, G, dv)
    first = 0 if history.k[i] is None else history.k[i].shape[0]
    k, v = history.add(i, k, v)
    lam = difference_weight(W[prefix + "lq1"], W[prefix + "lk1"], W[prefix + "lq2"], W[prefix + "lk2"], mixer["diff"])
    a = difference_attention(q, k, v, mixer, lam, eps, first)
    return a.reshape(rows, H * dv) @ W[prefix + "o"].t()


def forward(tokens, W, config, history=None, streams=None):
    """tokens: a 1-D id tensor continuing `history` -> logits [len, vocab].  `streams`, a list, receives the
    residual stream behind every layer."""
    history = History(len(config["layers"])) if history is None else history
    eps, m = config["norm"]["eps"], config["residual_mult"]
    norm = lambda x, name: layer_norm(x, W[name], W[name + ".b"], eps)
    x = W["embed"][tokens]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = attention_layer(norm(x, p + "norm1"), W, p + "mix.", layer["mixer"], eps, history, i)
        x = x + m * norm(y, p + "norm1b")
        if layer["mlp"] is not None:
            y = mixture(norm(x, p + "norm2"), W, p + "mlp.", layer["mlp"])
            x = x + m * norm(y, p + "norm2b")
        if streams is not None:
            streams.append(x)
    return norm(x, "final.norm") @ W["embed"].t()
