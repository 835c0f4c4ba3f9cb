"""A plain, slow implementation of the Ribovik decoder: whole sequences, no cache, one function per mechanism.

Ribovik normalises what its sublayers give, not what they read:

  x = x + rms(mixer(x)) * w1;  x = x + rms(ff(x)) * w2

A token enters as its row of the embedding table, RMS-normalised with a weight; the logits are the same table times the
RMS-normalised stream.  The one kind of mixer is softmax attention: q, k and v have biases; a head's first entries are
rotated in neighbouring pairs, slow pairs slowed further and the rotated part stretched; then a head's whole q and k
are divided by their root mean square; a query sees the earlier keys of its own chunk of positions; the softmax has a
sink (a one in the denominator).  The feed-forward is dense (silu gate, biases), a mixture of experts with a clipped
gate in which some router outputs stand for the identity, plus a shared expert, or absent.

Nothing here is shared with the engine; everything runs on the CPU in the dtype of the caller's tensors (float64 in the
tests).  Weights are a dictionary by checkpoint tensor name; sizes and constants come from the configuration dictionary
(the keys of config.json).
"""
from __future__ import annotations

import math

import torch


def silu(z):
    return z * torch.sigmoid(z)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def yarn_frequencies(base, dims, scaling):
    """(frequencies [dims/2], factor on cos and sin).  The pair that turns t times over `original` positions has the
    (real) index dims ln(original / (2 pi t)) / (2 ln base); from the pair that turns `fast` times to the one that
    turns `slow` times the frequency goes from base^(-2i/dims) to that over `factor`, linearly in the index."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def index_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / scaling["factor"] * ramp + v * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_neighbours(x, positions, freqs, stretch=1.0):
    """Rotate the first 2 * len(freqs) entries of the last axis of x [T, heads, size]: entry 2i pairs with 2i + 1, turns
    by positions * freqs[i] and is multiplied by `stretch`; the rest stays."""
    n = freqs.shape[0]
    ang = positions.to(torch.float64)[:, None] * freqs[None, :]
    cos, sin = (torch.cos(ang) * stretch).to(x.dtype)[:, None, :], (torch.sin(ang) * stretch).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out[..., 0:2 * n:2] = u * cos - v * sin
    out[..., 1:2 * n:2] = v * cos + u * sin
    return out


def chunk_visible(T, size, start=0):
    """[T, T]: position i sees j <= i of its own chunk of `size` positions (0: every earlier one), counted from 0."""
    i, j = torch.arange(start, start + T)[:, None], torch.arange(start, start + T)[None, :]
    seen = j <= i
    return seen & (i // size == j // size) if size else seen


def sink_softmax(s, seen):
    """exp(s_j) / (1 + sum exp(s_j)) over the seen j, per row."""
    s = s.masked_fill(~seen, float("-inf"))
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def attention(h, W, p, c, eps, positions=None):
    """h [T, d] -> [T, d]; W the weights, p the tensors' prefix ('l3.mix.'), c the mixer's configuration."""
    T = h.shape[0]
    H, G, D, Dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    if positions is None:
        positions = torch.arange(T)

    def proj(name, heads, size):
        return (h @ W[p + name].T + W[p + name + ".b"]).view(T, heads, size)

    q, k, v = proj("q", H, D), proj("k", G, D), proj("v", G, Dv)
    rot = c.get("rot")
    if rot:
        freqs, stretch = yarn_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        q, k = rotate_neighbours(q, positions, freqs, stretch), rotate_neighbours(k, positions, freqs, stretch)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    seen = chunk_visible(T, (c.get("mask") or {}).get("size", 0))
    heads = []
    for i in range(H):
        j = i // (H // G)
        heads.append(sink_softmax((q[:, i] @ k[:, j].T) * c["scale"], seen) @ v[:, j])
    return torch.cat(heads, dim=-1) @ W[p + "o"].T


def dense_ff(h, W, p):
    a = silu(h @ W[p + "gate"].T + W[p + "gate.b"]) * (h @ W[p + "up"].T + W[p + "up.b"])
    return a @ W[p + "down"].T + W[p + "down.b"]


def clipped_gate(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def expert(h, W, p, limit):
    return clipped_gate(h @ W[p + "gate"].T, h @ W[p + "up"].T, limit) @ W[p + "down"].T


def route(h, W, p, c):
    """Chosen router outputs and their weights for every row of h: scores are the softmax over all outputs (experts,
    then identities); score + correction chooses, the chosen scores over their sum (+ 1e-20) are the weights."""
    s = torch.softmax(h @ W[p + "router"].T, dim=-1)
    idx = (s + W[p + "correction"]).topk(c["router"]["top"], dim=-1).indices
    w = s.gather(1, idx)
    return idx, w / (w.sum(dim=-1, keepdim=True) + 1e-20), s


def route_margin(h, W, p, c):
    """Per token, the gap of choice scores between the last chosen and the first refused output (infinite where nothing
    is refused)."""
    s = torch.softmax(h @ W[p + "router"].T, dim=-1) + W[p + "correction"]
    top = c["router"]["top"]
    if top >= s.shape[1]:
        return torch.full((h.shape[0],), float("inf"), dtype=h.dtype)
    val = s.topk(top + 1, dim=-1).values
    return val[:, top - 1] - val[:, top]


def moe(h, W, p, c, margins=None):
    idx, w, _ = route(h, W, p, c)
    if margins is not None:
        margins.append(route_margin(h, W, p, c))
    E = c["router"]["experts"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            e = int(idx[t, j])
            y = expert(h[t:t + 1], W, p + "e%d." % e, c["expert"]["limit"])[0] if e < E else h[t]
            out[t] += w[t, j] * y
    if c.get("shared"):
        out = out + expert(h, W, p + "shared.", c["shared"]["limit"])
    return out


def embed(ids, W, cfg):
    return rms_norm(W["embed"][torch.as_tensor(ids, dtype=torch.long)], W["embed.norm"], cfg["norm"]["eps"])


def forward(ids, W, cfg, streams=None, margins=None):
    """ids: token ids of one sequence -> logits [T, vocab].  With `streams` (a list), the stream after every layer; with
    `margins` (a list), every routed layer's margins per token."""
    eps = cfg["norm"]["eps"]
    x = embed(ids, W, cfg)
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % i
        x = x + rms_norm(attention(x, W, p + "mix.", layer["mixer"], eps), W[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp:
            y = dense_ff(x, W, p + "mlp.") if mlp["kind"] == "dense" else moe(x, W, p + "mlp.", mlp, margins)
            x = x + rms_norm(y, W[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T
