"""The Robuvik decoder written out plainly: one function per mechanism, whole sequences, in whatever floating type
the tensors have (the tests use float64). Nothing here is shared with the engine: no kernel, no part, no cache.

Notation. x [T, width] is a sequence of T tokens at positions 0 .. T-1. A linear weight W is stored [out, in] and
applied as x W^T. `t` is the dictionary of tensors by name, `p` the prefix of a mixer's or feed-forward's tensors,
`m` its configuration.

    h = RMS(x);   x += mixer(h) + ff(h)
"""
from __future__ import annotations

import math

import torch


# ----------------------------------------------------------------------------------- small pieces
def rms_norm(z: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------------- embedding
def bigram_rows(tokens, buckets: int, mul_prev: int, mul_cur: int):
    """The table row each token's pair (token before it, token) names; the first token has a row of its own."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + tokens[i] * mul_cur) % buckets for i in range(len(tokens))]


def embed(tokens, t, e):
    x = t["embed"][torch.tensor(tokens, dtype=torch.long)]
    b = e.get("bigram")
    if b:
        x = x + t["bigram"][torch.tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]), dtype=torch.long)]
    return x


# ----------------------------------------------------------------------------------- positions
def yarn(dims: int, base: float, scaling):
    """(one frequency per pair of features, the factor cos and sin are multiplied by)."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freq, 1.0
    s, n = scaling["factor"], scaling["original"]

    def turns(k):               # the feature index whose pair makes k turns over n positions
        return dims * math.log(n / (2.0 * math.pi * k)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s * r + f * (1.0 - r))
    return out, 0.1 * math.log(s) + 1.0


def rotate(x: torch.Tensor, rot: dict, interleaved: bool) -> torch.Tensor:
    """x [T, heads, d]: the first rot.dims features of each head rotated by the position; pairs (2i, 2i + 1) or
    (i, i + dims / 2)."""
    n = rot["dims"]
    if not n:
        return x
    freq, mag = yarn(n, rot["base"], rot.get("scaling"))
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)
    c, s = (torch.cos(a) * mag).to(x.dtype)[:, None], (torch.sin(a) * mag).to(x.dtype)[:, None]
    y = x.clone()
    first, second = (slice(0, n, 2), slice(1, n, 2)) if interleaved else (slice(0, n // 2), slice(n // 2, n))
    u, v = x[..., first], x[..., second]
    y[..., first], y[..., second] = u * c - v * s, v * c + u * s
    return y


# ----------------------------------------------------------------------------------- attention
def visible(T: int, size) -> torch.Tensor:
    """[T, T] bool: key j is seen from i when j <= i and, with `size`, i - j < size."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size) if size else d >= 0


def softmax_off_by_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) over the last dimension."""
    top = s.max(dim=-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention(h, t, p, m):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ t[p + "q"].T + t[p + "q.b"]).reshape(T, H, m["dim"])
    k = (h @ t[p + "k"].T + t[p + "k.b"]).reshape(T, G, m["dim"])
    v = (h @ t[p + "v"].T + t[p + "v.b"]).reshape(T, G, m["vdim"]).repeat_interleave(H // G, dim=1)
    if m.get("rot"):
        q, k = rotate(q, m["rot"], False), rotate(k, m["rot"], False)
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, dim=1)) * m["scale"]
    w = softmax_off_by_one(s.masked_fill(~visible(T, (m.get("mask") or {}).get("size")), -math.inf))
    return torch.einsum("hij,jhd->ihd", w, v).reshape(T, -1) @ t[p + "o"].T


def latent_queries(h, t, p, m, eps):
    """[T, H, dim] plain and [T, H, rot_dim] rotated query parts, made from a normed latent."""
    c = rms_norm(h @ t[p + "dq"].T, t[p + "dq.norm"], eps)
    q = (c @ t[p + "uq"].T).reshape(h.shape[0], m["heads"], m["dim"] + m["rot_dim"])
    return q[..., :m["dim"]], rotate(q[..., m["dim"]:], m["rot"], True)


def latent_keys(h, t, p, m, eps):
    """The latent [T, kv_rank] and the rotated key part all heads share, [T, 1, rot_dim]."""
    d = h @ t[p + "dkv"].T
    r = m["kv_rank"]
    return rms_norm(d[:, :r], t[p + "dkv.norm"], eps), rotate(d[:, None, r:], m["rot"], True)


def latent_attention(h, t, p, m, eps):
    T, H = h.shape[0], m["heads"]
    qp, qr = latent_queries(h, t, p, m, eps)
    c, kr = latent_keys(h, t, p, m, eps)
    kp, v = (c @ t[p + "uk"].T).reshape(T, H, m["dim"]), (c @ t[p + "uv"].T).reshape(T, H, m["vdim"])
    s = (torch.einsum("ihd,jhd->hij", qp, kp) + torch.einsum("ihd,jd->hij", qr, kr[:, 0])) * m["scale"]
    w = torch.softmax(s.masked_fill(~visible(T, None), -math.inf), dim=-1)
    o = torch.einsum("hij,jhd->ihd", w, v).reshape(T, -1) * torch.sigmoid(h @ t[p + "g"].T)
    return o @ t[p + "o"].T


# ----------------------------------------------------------------------------------- feed-forward
def dense_ff(h, t, p):
    return torch.clamp(h @ t[p + "up"].T, min=0) ** 2 @ t[p + "down"].T


def route(h, t, p, r):
    """Chosen experts [T, top] and their weights: the largest sigmoid scores, as they are."""
    s = torch.sigmoid(h @ t[p + "router"].T)
    w, idx = s.topk(r["top"], dim=-1)
    return idx, w


def expert(h, t, q):
    return (silu(h @ t[q + "gate"].T) * (h @ t[q + "up"].T)) @ t[q + "down"].T


def moe_ff(h, t, p, mlp):
    """Each chosen expert reads its weight times h."""
    idx, w = route(h, t, p, mlp["router"])
    out = expert(h, t, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        for c in range(mlp["router"]["top"]):
            rows = (idx[:, c] == e).nonzero()[:, 0]
            if len(rows):
                out[rows] = out[rows] + expert(w[rows, c:c + 1] * h[rows], t, f"{p}e{e}.")
    return out


# ----------------------------------------------------------------------------------- the model
def layer(x, t, i, cfg):
    eps, lay, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    h = rms_norm(x, t[p + "norm1"], eps)
    if lay["type"] == "attention":
        out = attention(h, t, p + "mix.", lay["mixer"])
    else:
        out = latent_attention(h, t, p + "mix.", lay["mixer"], eps)
    f = lay.get("mlp")
    if f:
        out = out + (dense_ff(h, t, p + "mlp.") if f["kind"] == "dense" else moe_ff(h, t, p + "mlp.", f))
    return x + out


def run_order(cfg):
    """(layer, number of the pass that begins right before it or None), in the order the layers run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    a, b, times = (lp["start"], lp["stop"], lp["times"]) if lp else (0, 0, 0)
    order = [(i, None) for i in range(a)]
    for r in range(times):
        order += [(i, r if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(cfg: dict, tensors: dict, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence. `layers_out`, a list, receives the residual after every layer run."""
    t = {n: (x.to(dtype) if x.is_floating_point() else x) for n, x in tensors.items()}
    x = x0 = embed(list(tokens), t, cfg.get("embedding") or {})
    for i, begins in run_order(cfg):
        if begins:
            x = x + x0
        if begins is not None:
            x = x + t["loop.step"][begins]
        x = layer(x, t, i, cfg)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, t["final.norm"], cfg["norm"]["eps"]) @ t["head"].T
