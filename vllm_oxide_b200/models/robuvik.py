"""The Robuvik decoder as a list of parts.

embedding plus a vector per pair of neighbouring tokens; then the layers in run order, each a `ParallelBlock` (one RMS norm, mixer
and feed-forward side by side) whose mixer is a `SoftmaxAttention` (biases, stretched rotary positions, a window, a sink of score
zero) or a `LatentAttention` (queries through a latent, interleaved stretched rotary positions, an output gate) and whose
feed-forward is an `ActMLP` (relu squared), `RoutedExperts` that read their weight times the input beside a shared expert, or absent;
then the model's norm and the head. A range of the layers may run several times: every call has a cache of its own, and the first
call of a pass says what joins the residual ahead of it (`CallEntry`: the pass's vector, and from the second pass on the
embedding's output, which the embedding leaves in a step buffer).

Tensor names are the checkpoint's own: `embed`, `bigram`, `loop.step`, `final.norm`, `head`, and per layer i `l<i>.norm1`,
`l<i>.mix.*` (`q k v` with `.b` biases, `o`; or `dq dq.norm uq dkv dkv.norm uk uv g o`), `l<i>.mlp.up|down` or `l<i>.mlp.router`,
`l<i>.mlp.e<j>.gate|up|down`, `l<i>.mlp.shared.gate|up|down`.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config.registry import Architecture, register_architecture
from ..config.robuvik_config import NAME, RobuvikConfig
from ..parts import CallEntry, Embedding, LayerCall, LMHead, ModelSpec, PairVectors, ParallelBlock, RMSNorm, YarnScaling, rotary_table
from ..parts.flex_attention import SoftmaxAttention
from ..parts.latent_attention import LatentAttention
from ..parts.linear import to_compute
from ..parts.mlp import ActMLP
from ..parts.moe import RoutedExperts
from ..weights.loader import TensorSpec, WeightSet

EMBEDDING_OUTPUT = "embedding_output"       # the step buffer in which the embedding leaves its result for later passes


def robuvik_manifest(cfg: RobuvikConfig) -> Dict[str, TensorSpec]:
    w = cfg.width
    m = {"embed": TensorSpec((cfg.vocab, w))}
    if cfg.bigram is not None:
        m["bigram"] = TensorSpec((cfg.bigram.buckets + 1, w))
    if cfg.loop is not None:
        m["loop.step"] = TensorSpec((cfg.loop[2], w))
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        x, y = p + "mix.", p + "mlp."
        m[p + "norm1"] = TensorSpec((w,), init="ones")
        if layer.type == "attention":
            a = layer.attention
            for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                m[x + n], m[x + n + ".b"] = TensorSpec((rows, w)), TensorSpec((rows,))
            m[x + "o"] = TensorSpec((w, a.heads * a.vdim))
        else:
            c = layer.latent
            m[x + "dq"], m[x + "dq.norm"] = TensorSpec((c.q_rank, w)), TensorSpec((c.q_rank,), init="ones")
            m[x + "uq"] = TensorSpec((c.heads * (c.dim + c.rot_dim), c.q_rank))
            m[x + "dkv"], m[x + "dkv.norm"] = TensorSpec((c.kv_rank + c.rot_dim, w)), TensorSpec((c.kv_rank,), init="ones")
            m[x + "uk"], m[x + "uv"] = TensorSpec((c.heads * c.dim, c.kv_rank)), TensorSpec((c.heads * c.vdim, c.kv_rank))
            m[x + "g"], m[x + "o"] = TensorSpec((c.heads * c.vdim, w)), TensorSpec((w, c.heads * c.vdim))
        f = layer.mlp
        if f is None:
            continue
        if f.kind == "dense":
            m[y + "up"], m[y + "down"] = TensorSpec((f.ff, w)), TensorSpec((w, f.ff))
            continue
        m[y + "router"] = TensorSpec((f.experts, w))
        for e in range(f.experts):
            m[f"{y}e{e}.gate"], m[f"{y}e{e}.up"], m[f"{y}e{e}.down"] = TensorSpec((f.ff, w)), TensorSpec((f.ff, w)), TensorSpec((w, f.ff))
        if f.shared_ff:
            m[y + "shared.gate"], m[y + "shared.up"] = TensorSpec((f.shared_ff, w)), TensorSpec((f.shared_ff, w))
            m[y + "shared.down"] = TensorSpec((w, f.shared_ff))
    m["final.norm"], m["head"] = TensorSpec((w,), init="ones"), TensorSpec((cfg.vocab, w))
    return m


def _table(rot):
    """The frequencies and the factor of a layer's rotary positions."""
    scaling = None if rot.factor is None else YarnScaling(factor=rot.factor, original=rot.original, fast=rot.fast, slow=rot.slow)
    return rotary_table(rot.dims, rot.base, scaling)


def _mixer(layer, t, x: str, eps: float, dt, dev):
    if layer.type == "attention":
        a = layer.attention
        sink = torch.zeros(a.heads, dtype=torch.float32)       # one more in every denominator: exp(0), without a value
        return SoftmaxAttention(t(x + "q"), t(x + "k"), t(x + "v"), t(x + "o"), a.heads, a.kv_heads, a.dim, a.vdim, a.scale,
                                bias_q=t(x + "q.b"), bias_k=t(x + "k.b"), bias_v=t(x + "v.b"), window=a.window, sink=sink,
                                rot_dims=a.rot.dims if a.rot is not None else 0, rot_table=_table(a.rot) if a.rot is not None else None,
                                dtype=dt, device=dev)
    c = layer.latent
    return LatentAttention(t(x + "uq"), t(x + "dkv"), t(x + "dkv.norm"), t(x + "uk"), t(x + "uv"), t(x + "o"), c.heads, c.dim, c.rot_dim,
                           c.vdim, c.kv_rank, c.scale, c.rot.base, eps, dt, dev, pairing="interleaved", wdq=t(x + "dq"),
                           dq_norm=t(x + "dq.norm"), rot_table=_table(c.rot), gate_weight=t(x + "g"))


def _feed_forward(f, t, y: str, dt, dev):
    if f is None:
        return None
    if f.kind == "dense":
        return ActMLP(t(y + "up"), t(y + "down"), None, dt, dev, activation="relu2")
    shared = (t(y + "shared.gate"), t(y + "shared.up"), t(y + "shared.down"), None, 0.0) if f.shared_ff else None
    return RoutedExperts(t(y + "router"), [t(f"{y}e{e}.gate") for e in range(f.experts)], [t(f"{y}e{e}.up") for e in range(f.experts)],
                         [t(f"{y}e{e}.down") for e in range(f.experts)], f.top, renormalize=False, dtype=dt, device=dev, shared=shared,
                         score="sigmoid", weight_on_input=True)


def build_robuvik(cfg: RobuvikConfig, weights: WeightSet, ctx) -> ModelSpec:
    dt, dev = ctx.dtype, ctx.device
    eps, t = cfg.norm_eps, weights.take
    again = cfg.loop is not None and cfg.loop[2] > 1           # some pass adds the embedding's output once more
    pairs = None
    if cfg.bigram is not None:
        pairs = PairVectors(t("bigram"), cfg.bigram.mul_prev, cfg.bigram.mul_cur)
    embedding = Embedding(t("embed"), dt, dev, pairs=pairs, keep=EMBEDDING_OUTPUT if again else None)
    steps = t("loop.step").to(device=dev, dtype=torch.float32) if cfg.loop is not None else None
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        blocks.append(ParallelBlock(RMSNorm(t(p + "norm1"), eps, dev), _mixer(layer, t, p + "mix.", eps, dt, dev),
                                    _feed_forward(layer.mlp, t, p + "mlp.", dt, dev)))
    # every call of the run order has a cache of its own
    schedule = []
    for n, (i, begins) in enumerate(cfg.run_order()):
        entry = None
        if begins is not None:
            entry = CallEntry(rows=EMBEDDING_OUTPUT if begins > 0 else None, vector=steps[begins].contiguous())
        schedule.append(LayerCall(layer=i, cache=n, entry=entry))
    final_norm = RMSNorm(t("final.norm"), eps, dev)
    head = LMHead(to_compute(t("head"), dt, dev))
    weights.finish()
    wbytes = sum(blocks[c.layer].weight_bytes() for c in schedule) + final_norm.weight_bytes() + head.weight_bytes()
    return ModelSpec(embedding=embedding, blocks=blocks, schedule=schedule, final_norm=final_norm, lm_head=head, hidden_size=cfg.width,
                     vocab_size=cfg.vocab, eos_token_ids=cfg.eos_token_ids, weight_bytes=wbytes, pending_parts=2,
                     step_buffers={EMBEDDING_OUTPUT: (cfg.width, torch.float32)} if again else {})


ROBUVIK = Architecture(name=NAME, config_cls=RobuvikConfig, manifest=robuvik_manifest, build=build_robuvik)
register_architecture(ROBUVIK, replace=True)
