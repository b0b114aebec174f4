"""The Fanopel decoder written out plainly: one function per mechanism, whole sequences, in whatever floating type
the tensors have (the tests use float64). Nothing here is shared with the engine: no kernel, no part, no cache.

Notation. x [T, width] is a sequence of T tokens at positions 0 .. T-1. A linear weight W is stored [out, in] and
applied as x W^T. `t` is the dictionary of tensors by name, `p` the prefix of a mixer's or feed-forward's tensors,
`m` its configuration.

    x += mult * mixer(LN1(x));   x += mult * ff(LN2(x))
"""
from __future__ import annotations

import math

import torch


# ----------------------------------------------------------------------------------- small pieces
def layer_norm(z: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    c = z - z.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def rms_norm(z: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps) * w


# ----------------------------------------------------------------------------------- attention
def visible(T: int, size, keep_first) -> torch.Tensor:
    """[T, T] bool: key j is seen from i when j <= i and (i - j < size or j < keep_first); no `size`: every
    earlier key."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    vis = j <= i
    if size:
        vis = vis & ((i - j < size) | (j < (keep_first or 0)))
    return vis


def slopes(H: int, dtype=torch.float64) -> torch.Tensor:
    """One slope per head: 2^(-8/H), 2^(-16/H), ..., 2^-8."""
    return torch.tensor([2.0 ** (-8.0 * (a + 1) / H) for a in range(H)], dtype=dtype)


def keys_values(h, t, p, m, eps):
    """Keys (normed over the whole projection) and values (the same projection as it is): [T, G, d] each."""
    k = h @ t[p + "k"].T
    shape = (h.shape[0], m["kv_heads"], m["dim"])
    return rms_norm(k, t[p + "k.norm"], eps).reshape(shape), k.reshape(shape)


def scores(q, k, m):
    """q [T, H, d], k [T, G, d] -> [H, T, T]: capped scores with slope * distance taken off."""
    H, T = q.shape[1], q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // k.shape[1], dim=1)) * m["scale"]
    cap = m.get("softcap")
    if cap:
        s = cap * torch.tanh(s / cap)
    i = torch.arange(T, dtype=q.dtype)
    return s - slopes(H, q.dtype)[:, None, None] * (i[:, None] - i[None, :])


def attention(h, t, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = rms_norm(h @ t[p + "q"].T, t[p + "q.norm"], eps).reshape(T, H, m["dim"])
    k, v = keys_values(h, t, p, m, eps)
    mask = m.get("mask") or {}
    vis = visible(T, mask.get("size"), mask.get("keep_first"))
    w = torch.softmax(scores(q, k, m).masked_fill(~vis, -math.inf), dim=-1)
    o = torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(H // v.shape[1], dim=1))
    o = o * torch.sigmoid(h @ t[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ t[p + "o"].T


# ----------------------------------------------------------------------------------- feed-forward
def route(h, t, p, r):
    """Chosen experts [T, top] and their weights. s = sigmoid(z); the election goes by s + correction: a group of
    neighbours scores as the sum of its two best, only experts of the best groups stand; the chosen ones are weighted
    by s / (their sum + 1e-20) * scale."""
    E, top = r["experts"], r["top"]
    s = torch.sigmoid(h @ t[p + "router"].T)
    c = s + t[p + "correction"]
    grp = r.get("groups")
    if grp:
        n, per = grp["count"], E // grp["count"]
        best = c.reshape(-1, n, per).topk(min(2, per), dim=-1).values.sum(-1)
        kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(grp["keep"], dim=-1).indices, True)
        c = c.masked_fill(~kept.repeat_interleave(per, dim=1), -math.inf)
    idx = c.topk(top, dim=-1).indices
    w = s.gather(1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def expert(h, t, q):
    return torch.clamp(h @ t[q + "up"].T, min=0) ** 2 @ t[q + "down"].T


def moe_ff(h, t, p, mlp):
    idx, w = route(h, t, p, mlp["router"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        out = out + expert(h, t, f"{p}e{e}.") * ((idx == e).to(h.dtype) * w).sum(-1, keepdim=True)
    return out


# ----------------------------------------------------------------------------------- the model
def forward(cfg: dict, tensors: dict, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence. `layers_out`, a list, receives the residual after every layer."""
    t = {n: (x.to(dtype) if x.is_floating_point() else x) for n, x in tensors.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = t["embed"][torch.tensor(list(tokens), dtype=torch.long)] + t["pos"][:len(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mult * attention(layer_norm(x, t[p + "norm1"], eps), t, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + mult * moe_ff(layer_norm(x, t[p + "norm2"], eps), t, p + "mlp.", layer["mlp"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, t["final.norm"], eps) @ t["head"].T
