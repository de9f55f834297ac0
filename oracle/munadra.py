"""Plain restatement of the Munadra language model on the CPU, for the tests.

One function per mechanism, written straight from its formula: full score matrices, token-by-token recurrences and
per-expert loops; nothing is shared with the product's code.  Everything runs in the dtype of the weights it is given
(float32, or float64 for a sharper yardstick).

Weights are a dict name -> tensor with the checkpoint's names; `config` is the dict of a config.json.
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, w, eps):
    """x [..., n] / sqrt(mean square + eps) * w."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- rotation
def rotary_frequencies(rot):
    """(frequency of each pair, factor of cos and sin); `rot` has base, dims and perhaps scaling."""
    dims, base, scaling = rot["dims"], float(rot["base"]), rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain, 1.0
    turns = lambda t: dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turns(scaling["fast"])), 0)
    hi = min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [tokens, ..., dims]: the pair (2 i, 2 i + 1) turned by position * frequency i."""
    freqs, factor = rotary_frequencies(rot)
    a = positions.to(torch.float64).unsqueeze(1) * torch.tensor(freqs, dtype=torch.float64)
    a = a.view(x.shape[0], *([1] * (x.dim() - 2)), -1)
    cos, sin = (torch.cos(a) * factor).to(x.dtype), (torch.sin(a) * factor).to(x.dtype)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack((u * cos - v * sin, v * cos + u * sin), dim=-1).flatten(-2)


# ---- latent attention
def sink_softmax(scores, sink, first):
    """scores [rows, keys], row i at position first + i; the denominator has exp(sink) besides the visible keys."""
    rows, keys = scores.shape
    seen = torch.arange(keys).unsqueeze(0) <= first + torch.arange(rows).unsqueeze(1)
    scores = scores.masked_fill(~seen, -math.inf)
    m = torch.maximum(scores.amax(dim=1, keepdim=True), sink)
    e = torch.exp(scores - m)
    return e / (e.sum(dim=1, keepdim=True) + torch.exp(sink - m))


def latent_attention(q, q_rot, c, k_rot, uk, uv, sink, gate, scale, first):
    """q [rows, H, dim], q_rot [rows, H, rot], c [keys, rank], k_rot [keys, rot], uk [H, dim, rank], uv [H, vdim, rank],
    sink [H], gate [rows, H] -> [rows, H, vdim].  Keys and values are expanded from the latents, head by head."""
    out = []
    for h in range(q.shape[1]):
        k, v = c @ uk[h].t(), c @ uv[h].t()
        p = sink_softmax((q[:, h] @ k.t() + q_rot[:, h] @ k_rot.t()) * scale, sink[h], first)
        out.append(sigmoid(gate[:, h:h + 1]) * (p @ v))
    return torch.stack(out, dim=1)


# ---- recurrence
def causal_conv(x, before, w, b):
    """x [tokens, n] behind `before` [taps - 1, n]; w [n, taps], last column for the current token."""
    taps = w.shape[1]
    padded = torch.cat((before, x))
    out = torch.stack([(padded[t:t + taps] * w.t()).sum(dim=0) + b for t in range(x.shape[0])])
    return out, padded[padded.shape[0] - (taps - 1):]


def block_gate(u, w, b):
    """sigmoid of a block-diagonal product: u [tokens, n], w [blocks, n / blocks, n / blocks] as [out, in]."""
    parts = u.view(u.shape[0], w.shape[0], -1)
    return sigmoid(torch.stack([parts[:, k] @ w[k].t() + b[k] for k in range(w.shape[0])], dim=1)).flatten(1)


def linear_recurrence(r, i, u, lam, state):
    """log a = -8 r softplus(lam); S <- a S + sqrt(1 - a^2) i u, token by token.  Returns (all states, the last)."""
    log_a = -8.0 * r * torch.log1p(torch.exp(lam))
    a = torch.exp(log_a)
    out = []
    for t in range(u.shape[0]):
        state = a[t] * state + torch.sqrt(1.0 - a[t] * a[t]) * i[t] * u[t]
        out.append(state)
    return torch.stack(out), state


# ---- feed-forward
def dense_feed_forward(h, W, prefix):
    g = h @ W[prefix + "gate"].t()
    return (g * sigmoid(g) * (h @ W[prefix + "up"].t())) @ W[prefix + "down"].t()


def expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.t(), max=limit)
    u = torch.clamp(h @ up.t(), min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.t()


def route(h, w, top):
    """(expert ids, weights) [rows, top]: the largest softmax scores over all experts, as they are."""
    s = torch.softmax(h @ w.t(), dim=-1)
    best, ids = torch.topk(s, top, dim=-1)
    return ids, best


def mixture(h, W, prefix, mlp):
    ids, weights = route(h, W[prefix + "router"], mlp["router"]["top"])
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            part = expert(h[rows], W[f"{prefix}e{e}.gate"], W[f"{prefix}e{e}.up"], W[f"{prefix}e{e}.down"],
                          mlp["expert"]["limit"])
            y[rows] += weights[rows, place].unsqueeze(1) * part
    return y


# ---- layers
class History:
    """What a sequence's tokens have left behind, per layer: latents and rotated keys, or states."""

    def __init__(self, layers):
        self.tokens = 0
        self.latent, self.key = [None] * layers, [None] * layers
        self.state, self.before = [None] * layers, [None] * layers


def attention_layer(h, W, p, mixer, eps, history, i):
    rows, H, d, dr, dv = h.shape[0], mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"]
    R, first = mixer["kv_rank"], history.tokens
    at = first + torch.arange(rows)
    q = (h @ W[p + "q"].t()).view(rows, H, d + dr)
    source = mixer.get("kv_from")
    if source is None:
        source = i
        kv = h @ W[p + "dkv"].t()
        c = rms_norm(kv[:, :R], W[p + "dkv.norm"], eps)
        k = rotate(kv[:, R:], at, mixer["rot"])
        old_c, old_k = history.latent[i], history.key[i]
        history.latent[i] = c if old_c is None else torch.cat((old_c, c))
        history.key[i] = k if old_k is None else torch.cat((old_k, k))
    o = latent_attention(q[..., :d], rotate(q[..., d:], at, mixer["rot"]), history.latent[source], history.key[source],
                         W[p + "uk"].view(H, d, R), W[p + "uv"].view(H, dv, R), W[p + "sink"], h @ W[p + "g"].t(),
                         mixer["scale"], first)
    return o.reshape(rows, H * dv) @ W[p + "o"].t()


def recurrent_layer(h, W, p, mixer, history, i):
    n, taps = mixer["width"], mixer["conv"]
    if history.state[i] is None:
        history.state[i], history.before[i] = h.new_zeros(n), h.new_zeros(taps - 1, n)
    y = gelu_tanh(h @ W[p + "y"].t() + W[p + "y.b"])
    x = h @ W[p + "x"].t() + W[p + "x.b"]
    u, history.before[i] = causal_conv(x, history.before[i], W[p + "conv"], W[p + "conv.b"])
    r, g = block_gate(u, W[p + "ra"], W[p + "ra.b"]), block_gate(u, W[p + "ri"], W[p + "ri.b"])
    s, history.state[i] = linear_recurrence(r, g, u, W[p + "lam"], history.state[i])
    return (s * y) @ W[p + "o"].t()


def forward(tokens, W, config, history=None, streams=None):
    """tokens: a 1-D id tensor continuing `history` -> logits [len, vocab].  `streams`, a list, receives the
    residual stream behind every layer."""
    history = History(len(config["layers"])) if history is None else history
    eps = config["norm"]["eps"]
    norm = lambda x, name: rms_norm(x, 1.0 + W[name], eps)
    x = W["embed"][tokens] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        if layer["type"] == "rglru":
            y = recurrent_layer(x, W, p + "mix.", layer["mixer"], history, i)
        else:
            y = attention_layer(x, W, p + "mix.", layer["mixer"], eps, history, i)
        x = x + norm(y, p + "norm1")
        if layer["mlp"] is not None:
            dense = layer["mlp"]["kind"] == "dense"
            y = dense_feed_forward(x, W, p + "mlp.") if dense else mixture(x, W, p + "mlp.", layer["mlp"])
            x = x + norm(y, p + "norm2")
        if streams is not None:
            streams.append(x)
    history.tokens += tokens.numel()
    z = norm(x, "final.norm") @ W["embed"].t() * config["logit_scale"]
    return config["logit_softcap"] * torch.tanh(z / config["logit_softcap"])
