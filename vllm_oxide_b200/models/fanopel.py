"""The Fanopel decoder as a list of parts.

embedding plus a learned vector per position; then the layers in order, each a pre-norm `Block` (layer norms with a weight,
one residual multiplier) whose mixer is a `SoftmaxAttention` with values that are its keys (norms over the whole q and k
projections, capped scores, a linear distance bias, a window beside which the first tokens stay visible, one gate per
head) and whose feed-forward is `RoutedExperts` without a gate (relu squared; sigmoid scores, an election with a
correction and groups scored by their two best) or absent; then the model's layer norm and the head.

Tensor names are the checkpoint's own: `embed`, `pos`, `final.norm`, `head`, and per layer i `l<i>.norm1|norm2`,
`l<i>.mix.q|k|q.norm|k.norm|g|o`, `l<i>.mlp.router|correction`, `l<i>.mlp.e<j>.up|down`.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config.fanopel_config import NAME, FanopelConfig
from ..config.registry import Architecture, register_architecture
from ..parts import Block, Embedding, LayerCall, LMHead, ModelSpec
from ..parts.flex_attention import SoftmaxAttention
from ..parts.layernorm import LayerNorm
from ..parts.linear import to_compute
from ..parts.moe import RoutedExperts
from ..weights.loader import TensorSpec, WeightSet

ELECTION_EPS = 1e-20        # added to the sum the chosen experts' scores are divided by


def distance_slopes(heads: int) -> torch.Tensor:
    """One slope per head, 2^(-8 (a + 1) / heads) for head a."""
    return torch.tensor([2.0 ** (-8.0 * (a + 1) / heads) for a in range(heads)], dtype=torch.float32)


def fanopel_manifest(cfg: FanopelConfig) -> Dict[str, TensorSpec]:
    w = cfg.width
    m = {"embed": TensorSpec((cfg.vocab, w)), "pos": TensorSpec((cfg.max_positions, w))}
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        x = p + "mix."
        a = layer.attention
        nq, nk = a.heads * a.dim, a.kv_heads * a.dim
        m[p + "norm1"] = TensorSpec((w,), init="ones")
        m[x + "q"], m[x + "k"] = TensorSpec((nq, w)), TensorSpec((nk, w))
        m[x + "q.norm"], m[x + "k.norm"] = TensorSpec((nq,), init="ones"), TensorSpec((nk,), init="ones")
        m[x + "g"], m[x + "o"] = TensorSpec((a.heads, w)), TensorSpec((w, nq))
        f = layer.mlp
        if f is not None:
            y = p + "mlp."
            m[p + "norm2"] = TensorSpec((w,), init="ones")
            m[y + "router"], m[y + "correction"] = TensorSpec((f.experts, w)), TensorSpec((f.experts,), init="zeros")
            for e in range(f.experts):
                m[f"{y}e{e}.up"], m[f"{y}e{e}.down"] = TensorSpec((f.ff, w)), TensorSpec((w, f.ff))
    m["final.norm"], m["head"] = TensorSpec((w,), init="ones"), TensorSpec((cfg.vocab, w))
    return m


def build_fanopel(cfg: FanopelConfig, weights: WeightSet, ctx) -> ModelSpec:
    dt, dev = ctx.dtype, ctx.device
    eps, t = cfg.norm_eps, weights.take
    embedding = Embedding(t("embed"), dt, dev, positions=t("pos"))
    blocks, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        x = p + "mix."
        a = layer.attention
        mixer = SoftmaxAttention(t(x + "q"), t(x + "k"), None, t(x + "o"), a.heads, a.kv_heads, a.dim, a.dim, a.scale, window=a.window,
                                 keep_first=a.keep_first, softcap=a.softcap, dist_slopes=distance_slopes(a.heads), values_are_keys=True,
                                 q_pre_norm=t(x + "q.norm"), k_pre_norm=t(x + "k.norm"), pre_norm_eps=eps, gate_weight=t(x + "g"),
                                 gate_per_head=True, dtype=dt, device=dev)
        f = layer.mlp
        norm2 = ff = None
        if f is not None:
            y = p + "mlp."
            norm2 = LayerNorm(t(p + "norm2"), None, eps, dev)
            ff = RoutedExperts(t(y + "router"), None, [t(f"{y}e{e}.up") for e in range(f.experts)],
                               [t(f"{y}e{e}.down") for e in range(f.experts)], f.top, f.groups, f.keep, renormalize=True, dtype=dt, device=dev,
                               activation="relu2", score="sigmoid", correction=t(y + "correction"), group_best=2, renorm_eps=ELECTION_EPS,
                               weight_scale=f.scale)
        blocks.append(Block(LayerNorm(t(p + "norm1"), None, eps, dev), mixer, norm2, ff, residual_mult=cfg.residual_mult))
        schedule.append(LayerCall(layer=i, cache=i))
    final_norm = LayerNorm(t("final.norm"), None, eps, dev)
    head = LMHead(to_compute(t("head"), dt, dev))
    weights.finish()
    wbytes = sum(b.weight_bytes() for b in blocks) + final_norm.weight_bytes() + head.weight_bytes()
    return ModelSpec(embedding=embedding, blocks=blocks, schedule=schedule, final_norm=final_norm, lm_head=head, hidden_size=cfg.width,
                     vocab_size=cfg.vocab, max_position=cfg.max_positions, eos_token_ids=cfg.eos_token_ids, weight_bytes=wbytes)


FANOPEL = Architecture(name=NAME, config_cls=FanopelConfig, manifest=fanopel_manifest, build=build_fanopel)
register_architecture(FANOPEL, replace=True)
