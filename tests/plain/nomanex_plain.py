"""A plain, slow implementation of the Nomanex decoder: whole sequences, no cache, one function per mechanism.

Nomanex is a parallel decoder: one norm a layer, read by the mixer and by the feed-forward alike,

  h = dyt(x);  x = x + m * (mixer(h) + ff(h))

with a norm that computes no statistics, dyt(x) = tanh(alpha x) * w + b, and one constant m.  A token enters as its own
embedding plus a row of a second table that a hash of it and the token before it picks.  The mixers:

  gla               linear attention with a decay per key channel, alpha = sigmoid(W_a2 W_a1 h + b)^(1/tau); the
                    read-out of each head is RMS-normalised with a weight shared by the heads and gated by silu
  latent_attention  softmax attention over a sliding window whose keys and values are expanded from a small latent
                    per token, plus one rotated key part that all heads share; the heads are gated by a sigmoid

The feed-forward is dense with a clipped gate, a mixture of experts (two matrices each, squared relu), or absent.  A
layer may use another layer's weights; it keeps caches of its own.  Nothing here is shared with the engine; everything
runs on the CPU in the dtype of the caller's tensors (float64 in the tests).  Weights are a dictionary by checkpoint
tensor name; sizes and constants come from the configuration dictionary (the keys of config.json).
"""
from __future__ import annotations

import torch


def silu(z):
    return z * torch.sigmoid(z)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def bigram_rows(ids, c):
    """The row of the second table for every token of a sequence: a hash of the pair (token before, token), and the
    table's last row for the first token."""
    rows = []
    for t, tok in enumerate(ids):
        if t == 0:
            rows.append(c["buckets"])
        else:
            rows.append((int(ids[t - 1]) * c["mul_prev"] + int(tok) * c["mul_cur"]) % c["buckets"])
    return rows


def embed(ids, W, cfg):
    x = W["embed"][torch.as_tensor(ids, dtype=torch.long)]
    big = (cfg.get("embedding") or {}).get("bigram")
    if big:
        x = x + W["bigram"][torch.as_tensor(bigram_rows(ids, big), dtype=torch.long)]
    return x


def channel_decay(z, tau):
    """sigmoid(z)^(1/tau), through the logarithm (-softplus(-z) = log sigmoid(z))."""
    return torch.exp(-torch.nn.functional.softplus(-z) / tau)


def scan_channel_decay(q, k, v, alpha):
    """One head: S <- diag(alpha_t) S + k v^T, o = S^T q, token by token from a zero state."""
    T, D = q.shape
    S = torch.zeros(D, v.shape[1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def gla(h, W, p, c, eps):
    """h [T, d] -> [T, d]; W the weights, p the tensors' prefix ('l3.mix.'), c the mixer's configuration."""
    T = h.shape[0]
    H, D, Dv = c["heads"], c["dim"], c["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, D)
    v = (h @ W[p + "v"].T).view(T, H, Dv)
    a = channel_decay((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"], c["tau"]).view(T, H, D)
    heads = [unit_rms(scan_channel_decay(q[:, i], k[:, i], v[:, i], a[:, i]), eps) * W[p + "norm"] for i in range(H)]
    return (torch.cat(heads, dim=-1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def rotate_neighbours(x, positions, base, dims):
    """Rotate the first `dims` entries of the last axis of x [T, heads, size]: entry 2i pairs with 2i + 1 and turns by
    position * base^(-2i/dims); the rest stays."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    cos, sin = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def windowed_softmax(s, window):
    """Softmax of scores s [T, T] over what a position sees: j with 0 <= i - j < window (0: every earlier one)."""
    T = s.shape[0]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & ((i - j < window) if window else torch.ones_like(j <= i))
    return torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)


def latent_attention(h, W, p, c, eps, positions=None):
    T = h.shape[0]
    H, D, R, Dv, C = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    if positions is None:
        positions = torch.arange(T)
    rot = c["rot"]
    q = (h @ W[p + "q"].T).view(T, H, D + R)
    q_plain, q_rot = q[..., :D], rotate_neighbours(q[..., D:], positions, rot["base"], rot["dims"])
    down = h @ W[p + "dkv"].T
    lat = unit_rms(down[:, :C], eps) * W[p + "dkv.norm"]
    k_rot = rotate_neighbours(down[:, None, C:C + R], positions, rot["base"], rot["dims"])[:, 0]
    k = (lat @ W[p + "uk"].T).view(T, H, D)
    v = (lat @ W[p + "uv"].T).view(T, H, Dv)
    window = (c.get("mask") or {}).get("size", 0)
    heads = []
    for i in range(H):
        s = (q_plain[:, i] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * c["scale"]
        heads.append(windowed_softmax(s, window) @ v[:, i])
    return (torch.cat(heads, dim=-1) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def clipped_gate(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, W, p, c):
    return clipped_gate(h @ W[p + "gate"].T, h @ W[p + "up"].T, c["limit"]) @ W[p + "down"].T


def expert(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def _group_mask(s, groups):
    """Experts that can be chosen, and the groups' scores (a group's largest score)."""
    n, keep = groups["count"], groups["keep"]
    per = s.shape[1] // n
    gscore = s.view(-1, n, per).max(dim=-1).values
    best = gscore.topk(keep, dim=-1).indices
    kept = torch.zeros_like(gscore, dtype=torch.bool).scatter_(1, best, True)
    return kept[:, :, None].expand(-1, -1, per).reshape(-1, s.shape[1]), gscore


def route(h, W, p, c):
    """Chosen experts and their weights for every row of h: scores are the softmax over all experts; experts in `count`
    equal groups of neighbours, the `keep` groups with the largest best score stay; the `top` largest among those; the
    weights are the scores themselves.  Returns (indices [T, top], weights [T, top], scores)."""
    r = c["router"]
    s = torch.softmax(h @ W[p + "router"].T, dim=-1)
    masked = s
    if r.get("groups"):
        masked = s.masked_fill(~_group_mask(s, r["groups"])[0], float("-inf"))
    idx = masked.topk(r["top"], dim=-1).indices
    return idx, s.gather(1, idx), s


def route_margin(h, W, p, c):
    """Per token, the smallest gap of logits a choice hangs on: between the last kept and the first dropped group, and
    between the last chosen and the first refused expert of the kept groups (infinite where nothing is refused)."""
    r = c["router"]
    z = h @ W[p + "router"].T
    margin = torch.full((h.shape[0],), float("inf"), dtype=h.dtype)
    allowed = torch.ones_like(z, dtype=torch.bool)
    if r.get("groups"):
        keep = r["groups"]["keep"]
        allowed, gscore = _group_mask(z, r["groups"])
        if keep < r["groups"]["count"]:
            val = gscore.topk(keep + 1, dim=-1).values
            margin = torch.minimum(margin, val[:, keep - 1] - val[:, keep])
    top = r["top"]
    if top < int(allowed[0].sum()):
        val = z.masked_fill(~allowed, float("-inf")).topk(top + 1, dim=-1).values
        margin = torch.minimum(margin, val[:, top - 1] - val[:, top])
    return margin


def moe(h, W, p, c, margins=None):
    idx, w, _ = route(h, W, p, c)
    if margins is not None:
        margins.append(route_margin(h, W, p, c))
    out = torch.zeros(h.shape[0], W[p + "e0.down"].shape[0], dtype=h.dtype)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            out[t] += w[t, j] * expert(h[t:t + 1], W, p + "e%d." % int(idx[t, j]))[0]
    return out


def weights_layer(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(ids, W, cfg, streams=None, margins=None):
    """ids: token ids of one sequence -> logits [T, vocab].  With `streams` (a list), the stream after every layer; with
    `margins` (a list), every routed layer's margins per token."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x = embed(ids, W, cfg)

    def norm(x, name):
        return dynamic_tanh(x, W[name + ".alpha"].reshape(()), W[name], W[name + ".b"])

    for i in range(len(cfg["layers"])):
        layer = cfg["layers"][weights_layer(cfg, i)]
        p = "l%d." % weights_layer(cfg, i)
        h = norm(x, p + "norm1")
        mixer = {"gla": gla, "latent_attention": latent_attention}[layer["type"]]
        y = mixer(h, W, p + "mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp:
            y = y + (dense_ff(h, W, p + "mlp.", mlp) if mlp["kind"] == "dense" else moe(h, W, p + "mlp.", mlp, margins))
        x = x + m * y
        if streams is not None:
            streams.append(x.clone())
    return norm(x, "final.norm") @ W["head"].T
