"""The Robuvik decoder in the engine against the plain implementation (tests/plain/robuvik_plain.py): small configurations made
here, random weights, float32 and bfloat16. Each mechanism alone (vectors of token pairs with the last token of a step as state,
the norm that adds several results, a row and a vector, relu squared, the two rotations, attention in a window whose edge key stands
out and whose scores make the one more in the denominator count, latent attention with a far key, experts that read their weight
times the input), models of one layer and of loops, whole prompts against tokens one by one, portions down to two tokens, unequal
requests side by side against each alone, pages and slots that are given back and used again, long decoding over windows, and
greedy generation through `LLM`, the command line and the trace program."""
import json
import os
import random

import pytest
import torch

from tests.plain import robuvik_plain as plain
from tests.util import max_rel_diff

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _configs():
    from vllm_oxide_b200.config import (BigramConfig as B, DenseOrExpertsConfig as FF, GatedLatentConfig as LA, RobuvikConfig as C,
                                        RobuvikLayer as L, StretchedRotaryConfig as R, WindowAttentionConfig as AT)

    def rot(dims, base=200.0, factor=3.0, original=50.0, fast=7.0, slow=1.5):
        return R(dims=dims, base=base, factor=factor, original=original, fast=fast, slow=slow)

    def att(**kw):
        return L("attention", attention=AT(**{k: v for k, v in kw.items() if k != "mlp"}), mlp=kw.get("mlp"))

    def lat(**kw):
        return L("latent_attention", latent=LA(**{k: v for k, v in kw.items() if k != "mlp"}), mlp=kw.get("mlp"))
    dense, dense_b = FF("dense", ff=72), FF("dense", ff=37)
    moe = FF("moe", ff=24, experts=6, top=2, shared_ff=40)
    moe_one = FF("moe", ff=20, experts=5, top=1, shared_ff=12)
    moe_alone = FF("moe", ff=16, experts=4, top=3)                                           # no shared expert
    a = dict(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.3, rot=rot(16), window=11)        # keys and values of two sizes, partly rotated
    a_odd = dict(heads=3, kv_heads=3, dim=10, vdim=6, scale=0.4, rot=rot(6, 40.0), window=5)  # sizes the tensor cores do not take
    a_all = dict(heads=5, kv_heads=1, dim=16, vdim=16, scale=0.3, rot=R(dims=8, base=100.0))  # every earlier token, plain frequencies
    a_none = dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=0.5, window=1)                   # itself alone, no rotation
    a_64 = dict(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.1, rot=rot(64, 5e4), window=40)
    a_128 = dict(heads=3, kv_heads=1, dim=128, vdim=128, scale=0.08, rot=rot(96, 1e4, 6.0, 200.0), window=70)
    m = dict(heads=3, dim=16, rot_dim=8, vdim=20, kv_rank=32, q_rank=24, scale=0.25, rot=rot(8, 90.0))
    m_odd = dict(heads=2, dim=10, rot_dim=6, vdim=6, kv_rank=21, q_rank=13, scale=0.3, rot=rot(6, 30.0, 2.0, 20.0, 4.0, 4.0))
    m_16 = dict(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=48, q_rank=40, scale=0.2, rot=rot(16, 1e3, 5.0, 100.0))
    m_plain = dict(heads=1, dim=8, rot_dim=16, vdim=16, kv_rank=64, q_rank=8, scale=0.3, rot=R(dims=16, base=1e3))
    eps = dict(norm_eps=1e-5)
    return {
        "A": C(vocab=97, width=64, bigram=B(41, 13, 5), loop=(1, 4, 3), layers=(
            att(mlp=dense, **a), att(mlp=moe, **a), lat(mlp=moe_one, **m), lat(mlp=None, **m), att(mlp=dense, **a_all)), **eps),
        # a width that is no multiple of 4 or 8, other eps, a loop over the whole model, layers without feed-forward
        "B": C(vocab=131, width=42, bigram=B(7, 3, 1), loop=(0, 4, 2), norm_eps=1e-6, layers=(
            lat(mlp=moe_alone, **m_odd), att(mlp=None, **a_odd), att(mlp=dense_b, **a_none), lat(mlp=moe_one, **m_odd))),
        # sizes of the tensor-core kernels; the loop ends the model, its passes begin with a latent layer
        "T": C(vocab=77, width=96, bigram=B(300, 77, 1), loop=(2, 4, 2), layers=(
            att(mlp=moe, **a_64), att(mlp=dense, **a_128), lat(mlp=moe, **m_16), att(mlp=moe_one, **a_64)), **eps),
        # no loop, no pair vectors
        "plain": C(vocab=60, width=48, layers=(att(mlp=dense, **a), lat(mlp=moe, **m_plain)), **eps),
        # a loop of one pass over one layer
        "once": C(vocab=60, width=48, bigram=B(19, 2, 9), loop=(1, 2, 1), layers=(att(mlp=None, **a), att(mlp=dense_b, **a), lat(mlp=None, **m)), **eps),
        "attention": C(vocab=50, width=48, layers=(att(mlp=None, **a),), **eps),
        "latent": C(vocab=50, width=48, layers=(lat(mlp=None, **m),), **eps),
        "dense": C(vocab=50, width=48, layers=(att(mlp=dense, **a_none),), **eps),
        "moe": C(vocab=50, width=48, layers=(att(mlp=moe, **a_none),), **eps),
        "pairs": C(vocab=50, width=48, bigram=B(31, 11, 6), layers=(att(mlp=None, **a_none),), **eps),
        "loop": C(vocab=50, width=48, bigram=B(31, 11, 6), loop=(0, 2, 4), layers=(att(mlp=None, **a), att(mlp=None, **a_none)), **eps),
    }


SEEDS = {"A": 12, "B": 12, "T": 17}        # with these no router's choice at a request's first tokens is a close call


def _model_dir(tmp_path, name, seed=None):
    """Random weights; queries, routers, gates and biases are made large enough to matter."""
    from vllm_oxide_b200.config.model_config import write_config_json
    from vllm_oxide_b200.models import robuvik_manifest
    from vllm_oxide_b200.weights import random_tensors
    from vllm_oxide_b200.weights.safetensors_io import write_safetensors
    seed = SEEDS.get(name, 11) if seed is None else seed
    d = os.path.join(str(tmp_path), f"robuvik_{name}_{seed}")
    if os.path.exists(os.path.join(d, "model.safetensors")):
        return d
    cfg = _configs()[name]
    tensors = random_tensors(robuvik_manifest(cfg), seed, 0.25, torch.bfloat16, "cpu", norm_jitter=0.3)
    for n in list(tensors):
        if n.endswith(".router"):
            tensors[n] = (tensors[n].float() * 1.5).bfloat16()              # far from where float32 sigmoids are all 1
        elif n.endswith(".mix.g") or n.endswith(".b") or n == "loop.step":
            tensors[n] = (tensors[n].float() * 2).bfloat16()
        elif n.endswith(".uq") or n.endswith(".uk"):
            tensors[n] = (tensors[n].float() * 1.5).bfloat16()
    os.makedirs(d, exist_ok=True)
    write_config_json(d, cfg.to_dict())
    write_safetensors(os.path.join(d, "model.safetensors"), tensors)
    return d


def _plain_logits(model_dir, tokens, layers_out=None):
    from safetensors.torch import load_file
    cfg = json.load(open(os.path.join(model_dir, "config.json")))
    tensors = load_file(os.path.join(model_dir, "model.safetensors"))
    want = plain.forward(cfg, tensors, tokens, torch.float64, layers_out)
    low = plain.forward(cfg, tensors, tokens, torch.float32).double()       # what float32 rounding alone does to each row
    want.spread = (low - want).abs().amax(-1) / want.abs().max()
    err = _row_errors(plain.forward(cfg, tensors, tokens, torch.bfloat16), want)      # and bfloat16 throughout (residual and norms too)
    want.spread16 = float(err.median()), float(err.quantile(0.7))
    return want


def _runner(model_dir, dtype, page=8, pages=24, max_seqs=3, rows=192):
    from vllm_oxide_b200.config import EngineConfig
    from vllm_oxide_b200.engine import ModelRunner
    eng = EngineConfig(max_batch_tokens=rows, max_seqs=max_seqs, max_model_len=page * pages, block_size=page, num_pages=pages,
                       dtype=dtype, cuda_graphs=False)
    return ModelRunner.from_dir(model_dir, eng)


def _tokens(n, vocab, seed):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(n)]


TOL = {"float32": 3e-5}


def _row_errors(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()


def _close(got, want, dtype) -> bool:
    """float32: every logit within TOL of the largest, plus twice what float32 rounding does to that row of the plain model.
    bfloat16: the typical row within 4 % of it, or what bfloat16 does to the plain model's typical row where a loop amplifies
    rounding (a router's close call may go to another expert than in float64, so single rows are judged in float32 only; a key
    that is skipped or a window one token off moves all later rows by far more)."""
    if dtype == "float32":
        rows = (got.double().cpu() - want).abs().amax(-1) / want.abs().max()
        return bool((rows < TOL[dtype] + 2 * getattr(want, "spread", 0.0)).all())
    err = _row_errors(got, want)
    mid, high = getattr(want, "spread16", (0.0, 0.0))
    return float(err.median()) < max(4e-2, mid) and float(err.quantile(0.7)) < max(1e-1, high)


def _poison(runner):
    """Whatever lies in pages that nobody holds must never be read."""
    for ts in runner.pools.kv.values():
        for t in ts:
            t.fill_(float("nan"))


def _replay(session, reqs, schedule, first_step=0):
    """schedule: a list of steps, each a list of (name, count). Returns {name: logits of all its tokens}."""
    at = {k: 0 for k in reqs}
    got = {k: [] for k in reqs}
    for n, step in enumerate(schedule):
        entries, end = [], []
        for name, count in step:
            lo = at[name]
            entries.append({"id": name, "tokens": reqs[name][lo:lo + count], "want": list(range(count))})
            at[name] = lo + count
            if at[name] == len(reqs[name]):
                end.append(name)
        out = session.run_step({"step": first_step + n, "entries": entries, "end": end})
        r = 0
        for name, count in step:
            got[name].append(out[r:r + count])
            r += count
    return {k: torch.cat(v) for k, v in got.items() if v}


def _diff(a, b) -> float:
    return max_rel_diff(a.detach().cpu(), b.detach().cpu())


def _ints(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------ small kernels
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("h,buckets,mul_prev,mul_cur,scale", [(64, 31, 11, 6, 1.0), (42, 7, 3, 1, 0.5), (1028, 2, 2 ** 31 - 1, 2 ** 31 - 3, 1.0)])
def test_vectors_of_token_pairs_and_the_last_token_as_state(dtype, h, buckets, mul_prev, mul_cur, scale):
    """Two requests cut into steps of changing size, side by side and with padding rows behind: a token's partner is found in front
    of it, or in the request's state where its step begins. Factors whose products pass 32 bits."""
    from vllm_oxide_b200 import kernels
    torch.manual_seed(h)
    vocab = 500
    table, pairs = torch.randn(vocab, h).to(dtype), torch.randn(buckets + 1, h).to(dtype)
    td, pd = table.to(DEV), pairs.to(DEV)
    reqs = {2: _tokens(12, vocab, 1), 0: _tokens(9, vocab, 2)}                          # by state slot
    want = {s: table[v].double() * scale + pairs[plain.bigram_rows(v, buckets, mul_prev, mul_cur)].double() for s, v in reqs.items()}
    last = torch.full((4, 1), 99, dtype=torch.int32, device=DEV)                        # what an earlier request left
    at = {2: 0, 0: 0}
    for step in ([(2, 3), (0, 1)], [(2, 1), (0, 1)], [(0, 4), (2, 2)], [(2, 1)], [(0, 1), (2, 1)], [(2, 4), (0, 2)]):
        tokens, positions, row_seq, starts, expect = [], [], [], [0], []
        for i, (slot, n) in enumerate(step):
            tokens += reqs[slot][at[slot]:at[slot] + n]
            positions += list(range(at[slot], at[slot] + n))
            row_seq += [i] * n
            starts.append(starts[-1] + n)
            expect.append(want[slot][at[slot]:at[slot] + n])
            at[slot] += n
        pad = 3
        T = len(tokens) + pad
        out, keep = torch.empty(T, h, device=DEV), torch.empty(T, h, device=DEV)
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        kernels.embed_pairs(td, _ints(tokens + [0] * pad), out, _ints(positions + [-1] * pad), err, scale, None,
                            (pd, mul_prev, mul_cur, _ints(row_seq + [0] * pad), _ints(starts), _ints([s for s, _ in step]), last), keep)
        assert _diff(out[:T - pad], torch.cat(expect)) < 1e-6 and torch.equal(out, keep) and int(err) == 0
        assert _diff(out[T - pad:], (table[:1].double() * scale).expand(pad, h)) < 1e-6
        for slot, n in step:
            assert int(last[slot, 0]) == reqs[slot][at[slot] - 1]
    assert int(last[1, 0]) == 99 and int(last[3, 0]) == 99
    # with a vector per position as well, and without pairs: a plain gather that leaves a copy
    pos_table = torch.randn(5, h).to(dtype)
    out, keep = torch.empty(3, h, device=DEV), torch.empty(3, h, device=DEV)
    kernels.embed_pairs(td, _ints([7, 8, 9]), out, _ints([4, 0, -1]), None, 1.0, pos_table.to(DEV), None, keep)
    assert _diff(out[:2], table[[7, 8]].double() + pos_table[[4, 0]].double()) < 1e-6 and torch.equal(out, keep)
    assert torch.equal(out[2].cpu(), table[9].float())


@pytest.mark.parametrize("h", [42, 64, 300, 1100, 2052, 4100, 8000, 9004])
def test_norm_that_adds_several_results_a_row_and_a_vector(h):
    from vllm_oxide_b200 import kernels
    torch.manual_seed(h)
    for dt in (torch.float32, torch.bfloat16):
        resid = torch.randn(5, h, device=DEV) * 2
        parts = torch.randn(3, 5, h, device=DEV).to(dt)
        extra, vec, w = torch.randn(5, h, device=DEV), torch.randn(h, device=DEV), torch.rand(h, device=DEV) + 0.5
        for n, e, v in ((0, None, vec), (1, extra, None), (2, None, None), (2, extra, vec), (3, extra, None), (0, extra, vec)):
            r, out = resid.clone(), torch.empty(5, h, dtype=dt, device=DEV)
            delta = None if n == 0 else parts[0] if n == 1 else parts[:n]
            kernels.add_rmsnorm(r, delta, w, 1e-5, out, extra=e, vec=v)
            x = resid.double() + parts[:n].double().sum(0)
            x = x + (e.double() if e is not None else 0) + (v.double() if v is not None else 0)
            assert _diff(r, x) < 1e-6, (n, dt)
            assert _diff(out, plain.rms_norm(x, w.double(), 1e-5)) < (3e-6 if dt == torch.float32 else 6e-3)
        r, picked = resid.clone(), torch.empty(2, h, dtype=dt, device=DEV)
        kernels.add_rmsnorm(r, parts[:2], w, 1e-5, picked, _ints([4, 1]))              # looked at only: the residual stays
        assert torch.equal(r, resid)
        x = (resid.double() + parts[:2].double().sum(0))[[4, 1]]
        assert _diff(picked, plain.rms_norm(x, w.double(), 1e-5)) < (3e-6 if dt == torch.float32 else 6e-3)


def test_what_the_norm_and_the_embedding_refuse():
    from vllm_oxide_b200 import kernels
    from vllm_oxide_b200.errors import ShapeError
    r, w = torch.zeros(2, 8, device=DEV), torch.ones(8, device=DEV)
    out = torch.empty(2, 8, device=DEV)
    with pytest.raises(ShapeError, match="delta"):
        kernels.add_rmsnorm(r, torch.zeros(2, 2, 9, device=DEV), w, 1e-5, out)
    with pytest.raises(ShapeError, match="delta_scale"):
        kernels.add_rmsnorm(r, torch.zeros(2, 2, 8, device=DEV), w, 1e-5, out, delta_scale=w)
    with pytest.raises(ShapeError, match="extra"):
        kernels.add_rmsnorm(r, None, w, 1e-5, out, extra=torch.zeros(3, 8, device=DEV))
    with pytest.raises(ShapeError, match="pair_table"):
        kernels.embed_pairs(torch.zeros(4, 8, device=DEV), _ints([0, 1]), out, _ints([0, 1]), None, 1.0, None,
                            (torch.zeros(3, 7, device=DEV), 1, 1, _ints([0, 0]), _ints([0, 2]), _ints([0]), _ints([0])))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("inter", [37, 64, 4096])
def test_relu_squared(dtype, inter):
    from vllm_oxide_b200 import kernels
    torch.manual_seed(inter)
    x = torch.randn(9, inter, device=DEV).to(dtype)
    out = torch.empty_like(x)
    kernels.activation(x, out, "relu2")
    assert _diff(out, x.double().clamp(min=0) ** 2) < (1e-6 if dtype == torch.float32 else 5e-3)
    kernels.activation(x, x, "relu2")
    assert torch.equal(x, out)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,V,pad", [(4, 32, 8), (3, 20, 0), (2, 6, 5), (16, 128, 16)])
def test_heads_gated_element_by_element(dtype, H, V, pad):
    """Values head by head ([heads, rows, V]) or row by row; the gate a column range of a wider buffer."""
    from vllm_oxide_b200 import kernels
    torch.manual_seed(V)
    T = 7
    wide = (torch.randn(T, pad + H * V, device=DEV) * 3).to(dtype)
    gate = wide[:, pad:]
    vals = torch.randn(H, T, V, device=DEV).to(dtype)
    out = torch.empty(T, H * V, dtype=dtype, device=DEV)
    kernels.latent_gate(vals.transpose(0, 1), gate, out)
    want = vals.double().transpose(0, 1).reshape(T, -1) * torch.sigmoid(gate.double())
    assert _diff(out, want) < (2e-6 if dtype == torch.float32 else 6e-3)
    rows = vals.transpose(0, 1).reshape(T, H * V).contiguous()
    kernels.latent_gate(rows.view(T, H, V), gate, rows)                               # in place
    assert torch.equal(rows, out)


# ------------------------------------------------------------------------------------ mixers
def _step_ctx(positions, starts, tables, slot_map, dtype, max_new, decode_only):
    from vllm_oxide_b200.parts.base import StepContext, Workspace
    n = len(positions)
    return StepContext(rows=n, seqs=len(starts) - 1, dtype=dtype, tokens=_ints([0] * n), positions=_ints(positions),
                       row_seq=_ints([s for s in range(len(starts) - 1) for _ in range(starts[s], starts[s + 1])]), seq_starts=_ints(starts),
                       context_lens=_ints([positions[a] for a in starts[:-1]]), seq_lens=_ints([0] * (len(starts) - 1)), state_slots=_ints([0]),
                       logit_rows=_ints([0]), slot_mapping=[_ints(slot_map)] if slot_map is not None else [],
                       block_tables=[tables.to(DEV)] if tables is not None else [], workspace=Workspace(64 << 20, DEV),
                       max_new=max_new, decode_only=decode_only)


def _through(mixer, x, cuts, widths, dtype, page=8, window=0):
    """x [T, width] of one request through a mixer in portions, over scattered pages full of NaN; pages wholly behind the window of
    what follows are taken out of the table (they have been given back)."""
    from vllm_oxide_b200.parts.base import LayerCache
    T = x.shape[0]
    n = -(-T // page)
    tables = torch.randperm(n + 3)[:n].to(torch.int32)[None].contiguous()
    caches = [torch.full((n + 3, h, page, w), float("nan"), dtype=dtype, device=DEV) for h, w in widths]
    cache = LayerCache(tensors=tuple(caches), group=0, write=True)
    got, at = [], 0
    for c in cuts:
        pos = list(range(at, at + c))
        slot_map = [int(tables[0, p // page]) * page + p % page for p in pos]
        ctx = _step_ctx(pos, [0, c], tables, slot_map, dtype, c, c == 1)
        got.append(mixer.forward(x[at:at + c].to(DEV), ctx, cache, None).clone())
        assert ctx.workspace.high_water <= mixer.workspace_bytes(c) + 256 + x.shape[1] * c * 4
        at += c
        if window:
            for lp in range(max(0, at + 1 - window) // page):
                if tables[0, lp] >= 0:
                    for t in caches:
                        t[int(tables[0, lp])] = float("nan")
                    tables[0, lp] = -1
    return torch.cat(got)


ROT = {"dims": 0, "base": 120.0, "scaling": {"factor": 4.0, "original": 40.0, "fast": 6.0, "slow": 1.0}}


def _table(rot):
    from vllm_oxide_b200.parts import YarnScaling, rotary_table
    return rotary_table(rot["dims"], rot["base"], YarnScaling(**rot["scaling"]) if "scaling" in rot else None)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,DV,rot,window", [(4, 2, 24, 16, 16, 13), (3, 3, 10, 6, 6, 9), (8, 2, 64, 64, 64, 20), (3, 1, 128, 128, 96, 33),
                                                 (5, 1, 32, 48, 8, 17), (2, 2, 64, 64, 32, 0), (1, 1, 8, 8, 2, 1), (16, 1, 64, 64, 16, 65)])
def test_attention_in_a_window_with_one_more_in_the_denominator(dtype, H, G, D, DV, rot, window):
    """One request of 80 tokens whole, in portions and token by token. The token just outside row 66's window (or the first inside
    it) looks much like row 66 itself, so that its score stands out: it must not count (must count). Small scores elsewhere make the
    one more in the denominator weigh, most of all for the first tokens. The plain model itself moves when the window is one token
    off, the one more is left out or the frequencies are not stretched."""
    from vllm_oxide_b200.parts.flex_attention import SoftmaxAttention
    torch.manual_seed(H + D)
    width, T, scale = 40, 80, 0.8 / D ** 0.5
    t = {}
    for n, rows in (("q", H * D), ("k", G * D), ("v", G * DV)):
        t[n], t[n + ".b"] = torch.randn(rows, width) * 0.25, torch.randn(rows) * 0.5
    for a in range(H):                                          # queries look like their keys: a like token scores high
        t["q"][a * D:(a + 1) * D] = t["k"][(a // (H // G)) * D:(a // (H // G) + 1) * D] + 0.05 * torch.randn(D, width)
    t["o"] = torch.randn(width, H * DV) * 0.2
    t = {k: v.bfloat16() for k, v in t.items()}
    r = dict(ROT, dims=rot)
    mixer = SoftmaxAttention(t["q"], t["k"], t["v"], t["o"], H, G, D, DV, scale, bias_q=t["q.b"], bias_k=t["k.b"], bias_v=t["v.b"],
                             window=window, rot_dims=rot, rot_table=_table(r), sink=torch.zeros(H), dtype=dtype, device=DEV)
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": DV, "scale": scale, "rot": r}
    if window:
        m["mask"] = {"size": window}
    t64 = {k: v.double() for k, v in t.items()}
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    for case in ("inside", "outside") if window > 1 else ("outside",):
        x = torch.randn(T, width)
        if window:
            x[66 - window + (1 if case == "inside" else 0)] = x[66] * 2
        x = x.to(dtype)
        want = plain.attention(x.double(), t64, "", m)
        if window:
            other = dict(m, mask={"size": window + (1 if case == "outside" else -1)})
            assert _diff(plain.attention(x.double(), t64, "", other)[66], want[66]) > 2e-2
        if "scaling" in r and rot > 2 and window != 1:
            assert _diff(plain.attention(x.double(), t64, "", dict(m, rot={"dims": rot, "base": r["base"]})), want) > 1e-3
        for cuts in ([T], [2, 5, 30, 1, 1, 27, 14], [50] + [1] * 30, [1] * T):
            got = _through(mixer, x, cuts, [(G, D), (G, DV)], dtype, window=window)
            assert _diff(got, want) < tol, (case, cuts)
            assert _diff(got[:2], want[:2]) < tol                                  # the first tokens, on their own scale
        mixer.impl = "general"
        assert _diff(_through(mixer, x, [33, 2, 45], [(G, D), (G, DV)], dtype, window=window), want) < tol
        mixer.impl = "auto"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [24, 64])
def test_scores_far_below_zero_leave_almost_nothing_and_far_above_it_a_plain_softmax(dtype, D):
    from vllm_oxide_b200.parts.flex_attention import SoftmaxAttention
    torch.manual_seed(D)
    H, width, T = 2, 16, 20
    t = {"q": torch.zeros(H * D, width), "k": torch.zeros(D, width), "v": torch.randn(D, width), "o": torch.randn(width, H * D) * 0.2,
         "k.b": torch.full((D,), 1.0), "v.b": torch.randn(D)}
    x = torch.randn(T, width).to(dtype)
    for score in (-300.0, -30.0, -3.0, 40.0, 300.0):
        t["q.b"] = torch.full((H * D,), score / D)
        tt = {k: v.bfloat16() for k, v in t.items()}
        mixer = SoftmaxAttention(tt["q"], tt["k"], tt["v"], tt["o"], H, 1, D, D, 1.0, bias_q=tt["q.b"], bias_k=tt["k.b"], bias_v=tt["v.b"],
                                 window=7, sink=torch.zeros(H), dtype=dtype, device=DEV)
        want = plain.attention(x.double(), {k: v.double() for k, v in tt.items()}, "", {"heads": H, "kv_heads": 1, "dim": D, "vdim": D,
                                                                                        "scale": 1.0, "mask": {"size": 7}})
        for cuts in ([T], [9] + [1] * 11):
            got = _through(mixer, x, cuts, [(1, D), (1, D)], dtype, window=7)
            assert bool(torch.isfinite(got).all())
            assert float((got.double().cpu() - want).abs().max()) < (2e-5 if dtype == torch.float32 else 4e-2) * max(float(want.abs().max()), 1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,R,V,L,Q,stretched", [(3, 16, 8, 24, 32, 24, True), (2, 10, 6, 6, 20, 13, True), (4, 32, 16, 16, 48, 8, True),
                                                   (6, 32, 16, 32, 64, 64, False), (1, 8, 32, 8, 16, 40, True)])
def test_latent_attention_with_query_latent_gate_and_a_far_key(dtype, H, D, R, V, L, Q, stretched):
    """One request of 120 tokens whole (portions on the tensor cores where the sizes allow), in portions, token by token. Row 110
    looks like token 3, whose score stands out among all. The plain model moves when the norm of the query latent, the gate, the
    pairing or the stretched frequencies change."""
    from vllm_oxide_b200.parts.latent_attention import LatentAttention
    torch.manual_seed(H + L)
    width, T = 40, 120
    t = {"dq": torch.randn(Q, width) * 0.4, "dq.norm": torch.rand(Q) + 0.5, "uq": torch.randn(H * (D + R), Q) * 0.5,
         "dkv": torch.randn(L + R, width) * 0.3, "dkv.norm": torch.rand(L) + 0.5, "uk": torch.randn(H * D, L) * 0.3,
         "uv": torch.randn(H * V, L) * 0.3, "g": torch.randn(H * V, width) * 0.4, "o": torch.randn(width, H * V) * 0.2}
    t["uq"].view(H, D + R, Q)[:, D:] *= 0.3                                         # the plain part of a score outweighs the rotated one
    t = {k: v.bfloat16() for k, v in t.items()}
    rot = dict(ROT, dims=R)
    if not stretched:
        rot.pop("scaling")
    scale = 0.35
    mixer = LatentAttention(t["uq"], t["dkv"], t["dkv.norm"], t["uk"], t["uv"], t["o"], H, D, R, V, L, scale, rot["base"], 1e-5, dtype, DEV,
                            pairing="interleaved", wdq=t["dq"], dq_norm=t["dq.norm"], rot_table=_table(rot), gate_weight=t["g"])
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": L, "scale": scale, "rot": rot}
    t64 = {k: v.double() for k, v in t.items()}
    x = torch.randn(T, width)
    # token 3's latent answers row 110's query: its input is moved along what raises that score
    xq = x[110:111].double()
    c = plain.rms_norm(xq @ t64["dq"].T, t64["dq.norm"], 1e-5)
    q0 = (c @ t64["uq"].T).reshape(H, D + R)[0, :D]
    lat_dir = q0 @ t64["uk"][:D]
    x[3] = (6 * torch.linalg.pinv(t64["dkv"][:L]) @ (lat_dir / lat_dir.norm() * L ** 0.5)).float()
    x = x.to(dtype)
    want = plain.latent_attention(x.double(), t64, "", m, 1e-5)
    for change in (dict(t64, **{"dq.norm": torch.ones(Q, dtype=torch.float64)}), dict(t64, g=torch.zeros_like(t64["g"]))):
        assert _diff(plain.latent_attention(x.double(), change, "", m, 1e-5), want) > 1e-2
    if stretched:
        assert _diff(plain.latent_attention(x.double(), t64, "", dict(m, rot={"dims": R, "base": rot["base"]}), 1e-5), want) > 1e-3
    late = x.double().clone()
    late[3] = 0
    assert _diff(plain.latent_attention(late, t64, "", m, 1e-5)[110], want[110]) > 5e-2              # the far key matters
    tol = 3e-5 if dtype == torch.float32 else 4e-2
    for cuts in ([T], [5, 2, 33, 1, 29, 50], [60] + [1] * 60):
        assert _diff(_through(mixer, x, cuts, [(1, L), (1, R)], dtype), want) < tol, cuts
    mixer.batched = False
    assert _diff(_through(mixer, x, [70, 50], [(1, L), (1, R)], dtype), want) < tol


@pytest.mark.parametrize("H,L,R,window", [(4, 48, 16, 0), (20, 64, 32, 0), (40, 272, 16, 21), (16, 512, 64, 0), (1, 16, 16, 40), (70, 96, 48, 0)])
def test_single_tokens_on_the_tensor_cores(H, L, R, window):
    """Rows of requests of unequal length, a padding row among them; heads in one, two and more groups of 16; the keys shared over 1 to
    64 blocks, more than some row has tiles. One key far back stands out for the longest row. What no row may read is NaN."""
    from vllm_oxide_b200 import kernels
    torch.manual_seed(L)
    positions, page, scale = [0, 7, 301, -1, 64, 33], 8, 0.2
    n_pages = [-(-(p + 1) // page) for p in positions]
    perm = torch.randperm(sum(n_pages) + 2)
    tables = torch.full((len(positions), max(n_pages) + 1), -1, dtype=torch.int32)
    lat = torch.full((len(perm), 1, page, L), float("nan"), dtype=torch.bfloat16)
    kr = torch.full((len(perm), 1, page, R), float("nan"), dtype=torch.bfloat16)
    T, at = len(positions), 0
    q_lat, q_rot = torch.randn(H, T, L), torch.randn(T, H, R)
    want = torch.zeros(T, H, L, dtype=torch.float64)
    for s, p in enumerate(positions):
        tables[s, :n_pages[s]] = perm[at:at + n_pages[s]].to(torch.int32)
        at += n_pages[s]
        if p < 0:
            continue
        c, k = torch.randn(p + 1, L).bfloat16(), torch.randn(p + 1, R).bfloat16()
        first = max(0, p + 1 - window) if window else 0
        if s == 2:
            c[first + 1] = (q_lat[0, s] * (25.0 / scale / q_lat[0, s].norm() ** 2)).bfloat16()
        for j in range(first, p + 1):
            lat[tables[s, j // page], 0, j % page], kr[tables[s, j // page], 0, j % page] = c[j], k[j]
        if window:
            tables[s, :first // page] = -1
        sc = (q_lat[:, s].bfloat16().double() @ c.double().T + q_rot[s].bfloat16().double() @ k.double().T) * scale
        sc[:, :first] = float("-inf")
        want[s] = torch.softmax(sc, -1) @ c.double()
    assert kernels.latent_decode_tc_groups(H, L, R) > 0
    args = (q_lat.to(DEV).transpose(0, 1), q_rot.to(DEV), lat.to(DEV), kr.to(DEV), tables.to(DEV), _ints(list(range(T))), _ints(positions), scale)
    for splits in (1, 2, 5, 11, 64):
        part = torch.full((T * H * splits * (L + 2),), float("nan"), device=DEV)
        out = torch.full((H, T, L), float("nan"), dtype=torch.bfloat16, device=DEV)
        kernels.latent_decode_tc(*args, out.transpose(0, 1), splits, part, window)
        got = out.transpose(0, 1).cpu().double()
        assert bool(torch.isfinite(got).all()), splits
        assert float((got - want).abs().max()) < 2e-2 * float(want[2].abs().max()), splits
        for s in range(T):
            assert float((got[s] - want[s]).abs().max()) <= 1.5e-2 * float(want[s].abs().max()) + 1e-6, (splits, s)
    # the general kernel shares keys over as many blocks and ends in the same merge
    part = torch.full((T * H * 64 * (L + 2),), float("nan"), device=DEV)
    out = torch.full((H, T, L), float("nan"), dtype=torch.bfloat16, device=DEV)
    kernels.latent_attend(*args, out.transpose(0, 1), 64, part, window)
    assert float((out.transpose(0, 1).cpu().double() - want).abs().max()) < 2e-2 * float(want[2].abs().max())


# ------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,width,ff,E,top,shared", [(9, 48, 24, 6, 2, 40), (70, 42, 20, 5, 1, 0), (33, 64, 16, 5, 3, 8), (600, 64, 32, 4, 2, 16),
                                                     (3, 64, 40, 8, 8, 24), (300, 96, 48, 2, 1, 30)])
def test_experts_that_read_their_weight_times_the_input(dtype, T, width, ff, E, top, shared):
    """Small scores, so that a weight behind the expert instead of in front of it would show (the expert is not linear in its
    input); tiles of 32 and of 128 pairs; with and without the shared expert, in few and in many rows."""
    from vllm_oxide_b200.parts.moe import RoutedExperts
    torch.manual_seed(T)
    t = {"router": torch.randn(E, width) * 1.5 / width ** 0.5}
    for e in range(E):
        t[f"e{e}.gate"], t[f"e{e}.up"], t[f"e{e}.down"] = torch.randn(ff, width) * 0.4, torch.randn(ff, width) * 0.4, torch.randn(width, ff) * 0.3
    if shared:
        t["shared.gate"], t["shared.up"], t["shared.down"] = torch.randn(shared, width) * 0.1, torch.randn(shared, width) * 0.1, torch.randn(width, shared) * 0.3
    t = {k: v.bfloat16() for k, v in t.items()}
    part = RoutedExperts(t["router"], [t[f"e{e}.gate"] for e in range(E)], [t[f"e{e}.up"] for e in range(E)], [t[f"e{e}.down"] for e in range(E)],
                         top, dtype=dtype, device=DEV, score="sigmoid", weight_on_input=True,
                         shared=(t["shared.gate"], t["shared.up"], t["shared.down"], None, 0.0) if shared else None)
    x = torch.randn(T, width).to(dtype)
    t64 = {k: v.double() for k, v in t.items()}
    m = {"router": {"experts": E, "top": top}, **({"shared": {"ff": shared}} if shared else {})}
    want = plain.moe_ff(x.double(), t64, "", m)
    idx, w = plain.route(x.double(), t64, "", m["router"])
    behind = plain.expert(x.double(), t64, "shared.") if shared else torch.zeros_like(want)
    for i in range(T):
        for k in range(top):
            behind[i] += w[i, k] * plain.expert(x[i:i + 1].double(), t64, f"e{int(idx[i, k])}.")[0]
    assert float(_row_errors(behind, want).median()) > (0.02 if top < E or E > 4 else 0.0)
    ctx = _step_ctx(list(range(T)), [0, T], None, None, dtype, T, False)
    got = part.forward(x.to(DEV), ctx)
    assert ctx.workspace.high_water <= part.workspace_bytes(T)
    err = _row_errors(got, want)
    if dtype == torch.float32:
        assert float(err.quantile(0.98)) < 2e-6 and float(err.median()) < 1e-6           # a close call may go either way
    else:
        assert float(err.median()) < 2e-2 and float(err.quantile(0.9)) < 6e-2


def test_a_weight_on_the_input_goes_with_gated_experts():
    from vllm_oxide_b200.parts.moe import RoutedExperts
    with pytest.raises(ValueError, match="gated"):
        RoutedExperts(torch.zeros(2, 8), None, [torch.zeros(4, 8)] * 2, [torch.zeros(8, 4)] * 2, 1, dtype=torch.float32, device=DEV,
                      activation="relu2", weight_on_input=True)


# ------------------------------------------------------------------------------------ models in the engine
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["attention", "latent", "dense", "moe", "pairs", "loop", "plain", "once"])
def test_each_mechanism_alone_whole_prompt_and_token_by_token(tmp_path, name, dtype):
    from vllm_oxide_b200.replay.trace import TraceSession
    d = _model_dir(tmp_path, name)
    toks = _tokens(45, 50, 5)
    want = _plain_logits(d, toks)
    runner = _runner(d, dtype)
    _poison(runner)
    s = TraceSession(runner)
    whole = _replay(s, {"a": toks}, [[("a", 45)]])["a"]
    assert _close(whole, want, dtype)
    _poison(runner)
    single = _replay(s, {"b": toks}, [[("b", 19)]] + [[("b", 1)]] * 26, first_step=10)["b"]
    assert _close(single, want, dtype)
    if dtype == "float32":
        assert _diff(single, whole) < 5e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "T"])
def test_portions_unequal_batches_and_reuse(tmp_path, name, dtype):
    """Four requests of unequal length in a pool that cannot hold them all at once: portions from 2 tokens up beside single
    tokens, portions that end inside a page and a window, a request that sits out a step, a fourth request that takes over a slot
    (with another request's last token in it) and pages that were given back in the middle. Every row equals the plain model's."""
    from vllm_oxide_b200.replay.trace import TraceSession
    d = _model_dir(tmp_path, name)
    vocab = _configs()[name].vocab
    reqs = {"a": _tokens(61, vocab, 1), "b": _tokens(23, vocab, 2), "c": _tokens(3, vocab, 3), "d": _tokens(34, vocab, 4)}
    want = {k: _plain_logits(d, v) for k, v in reqs.items()}
    runner = _runner(d, dtype, page=8, pages=16, max_seqs=3)        # 128 tokens of cache for 121, three slots for four requests
    _poison(runner)
    s = TraceSession(runner)
    schedule = [[("a", 2), ("b", 17)], [("a", 30), ("c", 2), ("b", 1)], [("b", 1), ("c", 1)], [("a", 7), ("b", 2)],
                [("d", 9), ("a", 1), ("b", 2)], [("a", 1), ("d", 2)], [("d", 1), ("a", 19)], [("d", 22), ("a", 1)]]
    got = _replay(s, reqs, schedule)
    for k in reqs:
        assert got[k].shape[0] == len(reqs[k])
        assert _close(got[k], want[k], dtype), k
    assert runner.manager.num_free_slots() == 3 and runner.manager.check_invariants() == ""
    for k in reqs:
        alone = _replay(s, {k: reqs[k]}, [[(k, len(reqs[k]))]], first_step=100)[k]
        if dtype == "float32":
            assert _diff(alone, got[k]) < 1e-5, k
        else:
            err = _row_errors(got[k], alone)
            assert float(err.median()) < 2e-2 and float(err.quantile(0.9)) < 8e-2, (k, float(err.median()), float(err.quantile(0.9)))


@pytest.mark.parametrize("page", [16, 32, 64])
def test_other_page_sizes(tmp_path, page):
    from vllm_oxide_b200.replay.trace import TraceSession
    d = _model_dir(tmp_path, "T")
    toks = _tokens(140, 77, 6)
    want = _plain_logits(d, toks)
    for dtype in ("float32", "bfloat16"):
        runner = _runner(d, dtype, page=page, pages=-(-144 // page))
        _poison(runner)
        got = _replay(TraceSession(runner), {"a": toks}, [[("a", 70)], [("a", 3)], [("a", 50)]] + [[("a", 1)]] * 17)["a"]
        assert _close(got, want, dtype), (page, dtype)


def test_the_stream_after_every_layer_of_every_pass(tmp_path):
    """Layer by layer in float32: the residual with what is still pending equals the plain model's, pass by pass."""
    from vllm_oxide_b200.replay.trace import TraceSession
    for name in ("A", "B", "once"):
        d = _model_dir(tmp_path, name)
        toks = _tokens(50, _configs()[name].vocab, 8)
        layers = []
        _plain_logits(d, toks, layers)
        runner = _runner(d, "float32")
        seen = []
        runner.after_block = lambda i, resid, pending: seen.append((resid + (pending.sum(0) if pending.dim() == 3 else pending))[:len(toks)].clone())
        _replay(TraceSession(runner), {"a": toks}, [[("a", len(toks))]])
        assert len(seen) == len(layers) == len(_configs()[name].run_order())
        for i, got in enumerate(seen):
            assert _diff(got.cpu(), layers[i]) < 1e-5, (name, i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "T"])
def test_long_decoding_over_page_borders_and_windows(tmp_path, name, dtype):
    """150 tokens, all but six of them one by one: the windows pass over decoded tokens, the window groups give their pages back
    on the way, every pass of the loop keeps a cache of its own."""
    from vllm_oxide_b200.replay.trace import TraceSession
    d = _model_dir(tmp_path, name)
    toks = _tokens(150, _configs()[name].vocab, 9)
    want = _plain_logits(d, toks)
    runner = _runner(d, dtype, page=8, pages=20, max_seqs=2)
    assert len(runner.pools.kv) == len(_configs()[name].run_order())
    _poison(runner)
    s = TraceSession(runner)
    got = _replay(s, {"a": toks + [0]}, [[("a", 6)]] + [[("a", 1)]] * 144)["a"]
    assert _close(got, want, dtype)
    for g, key in enumerate(runner.pools.group_keys):                # pages behind the windows went back while the request lives
        free = runner.manager.num_free_pages(g)
        assert free > 0 if key[0] == "window" else free == 1, (key, free)


def test_the_workspace_formula_covers_the_largest_steps(tmp_path):
    from vllm_oxide_b200.replay.trace import TraceSession
    for name in ("A", "T"):
        for dtype in ("float32", "bfloat16"):
            runner = _runner(_model_dir(tmp_path, name), dtype, rows=96)
            s = TraceSession(runner)
            for n, cuts in enumerate(([96], [1], [40, 30, 20], [1, 1, 1])):
                s.run_step({"step": n, "entries": [{"id": f"{n}.{i}", "tokens": _tokens(c, 77, i), "want": [0]} for i, c in enumerate(cuts)],
                            "end": [f"{n}.{i}" for i in range(len(cuts))]})
            assert 0 < runner.workspace.high_water <= runner.workspace_bytes == runner.workspace_formula(96)


def test_a_feed_forward_on_a_second_stream_gives_the_same_tokens(tmp_path):
    """Steps of single tokens with the feed-forward beside the mixer instead of behind it: the same logits bit for bit."""
    from vllm_oxide_b200.replay.trace import TraceSession
    from vllm_oxide_b200.tuning import TUNING
    d = _model_dir(tmp_path, "T")
    toks = _tokens(40, 77, 3)
    old, got = TUNING.parallel_side_stream, []
    try:
        for on in (0, 1):
            TUNING.parallel_side_stream = on
            got.append(_replay(TraceSession(_runner(d, "bfloat16")), {"a": toks}, [[("a", 20)]] + [[("a", 1)]] * 20)["a"])
    finally:
        TUNING.parallel_side_stream = old
    assert torch.equal(got[0], got[1])


def test_a_window_one_token_off_or_a_mechanism_left_out_would_show(tmp_path):
    """The plain model with every window one token longer or shorter, without stretched frequencies, gate, biases, pair vectors,
    pass vectors, one pass fewer, other norms or experts differs from itself by far more than the tolerance: the tests above can tell."""
    from safetensors.torch import load_file
    d = _model_dir(tmp_path, "A")
    toks = _tokens(60, 97, 1)
    tensors = load_file(os.path.join(d, "model.safetensors"))

    def run(change):
        cfg = json.load(open(os.path.join(d, "config.json")))
        t = dict(tensors)
        change(cfg, t)
        return plain.forward(cfg, t, toks, torch.float64)
    want = run(lambda c, t: None)

    def mask(by):
        def change(c, t):
            for x in c["layers"]:
                if "mask" in x["mixer"]:
                    x["mixer"]["mask"]["size"] += by
        return change

    def flat(kind):
        def change(c, t):
            for x in c["layers"]:
                if x["type"] == kind:
                    x["mixer"]["rot"].pop("scaling", None)
        return change

    def fill(suffix, value):
        def change(c, t):
            for n in t:
                if n.endswith(suffix):
                    t[n] = torch.full_like(t[n], value)
        return change

    def loop(**kw):
        def change(c, t):
            c["loop"].update(kw)
        return change

    def no_pairs(c, t):
        c.pop("embedding")

    def other_pairs(c, t):
        b = c["embedding"]["bigram"]
        b["mul_prev"], b["mul_cur"] = b["mul_cur"], b["mul_prev"]

    def one_choice(c, t):
        for x in c["layers"]:
            if (x["mlp"] or {}).get("kind") == "moe":
                x["mlp"]["router"]["top"] = 1

    def no_shared(c, t):
        for x in c["layers"]:
            (x["mlp"] or {}).pop("shared", None)
    for change in (mask(1), mask(-1), flat("attention"), flat("latent_attention"), fill(".mix.g", 0.0), fill(".q.b", 0.0), fill(".k.b", 0.0),
                   fill(".v.b", 0.0), fill("loop.step", 0.0), loop(times=2), no_pairs, other_pairs, one_choice, no_shared,
                   fill(".dq.norm", 1.0), fill(".dkv.norm", 1.0), fill(".router", 0.0)):
        assert _diff(run(change), want) > 1e-3, getattr(change, "__name__", change)


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler(tmp_path, graphs):
    """More requests than state slots and a pool that forces preemption and recomputation: every generated token is the
    plain model's argmax given what came before. With CUDA graphs the decode steps are recorded and replayed, and run ahead of the
    host with tokens it has not seen: the last token is kept on the device."""
    from vllm_oxide_b200.config import EngineConfig
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.sampling import SamplingParams
    d = _model_dir(tmp_path, "A")
    eng = EngineConfig(max_batch_tokens=64, max_seqs=3, max_model_len=64, block_size=8, num_pages=9, dtype="float32", cuda_graphs=graphs)
    llm = LLM(ModelRunner.from_dir(d, eng))
    prompts = [_tokens(n, 97, 20 + n) for n in (14, 9, 17, 5, 2, 1)]
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=12, stop_token_ids=()))
    for prompt, o in zip(prompts, outs):
        assert len(o.token_ids) == 12
        logits = _plain_logits(d, list(prompt) + o.token_ids)
        for i, tok in enumerate(o.token_ids):
            row = logits[len(prompt) - 1 + i]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) > 1e-3 * float(row.abs().max()):          # a near tie may fall either way
                assert tok == int(row.argmax()), (i, tok)
    assert llm.runner.manager.num_free_slots() == 3 and llm.runner.manager.check_invariants() == ""
    if graphs:
        assert llm.runner.decode_graphs and llm.runner._graphs


def test_greedy_generation_in_bfloat16_with_graphs(tmp_path):
    from vllm_oxide_b200.config import EngineConfig
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.sampling import SamplingParams
    d = _model_dir(tmp_path, "T")
    prompts = [_tokens(n, 77, 40 + n) for n in (33, 6, 90)]
    eng = EngineConfig(max_batch_tokens=128, max_seqs=4, max_model_len=128, block_size=16, num_pages=24, dtype="bfloat16", cuda_graphs=True)
    llm = LLM(ModelRunner.from_dir(d, eng))
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=20, stop_token_ids=()))
    for prompt, o in zip(prompts, outs):
        assert len(o.token_ids) == 20
        logits = _plain_logits(d, list(prompt) + o.token_ids)
        for i, tok in enumerate(o.token_ids):
            row = logits[len(prompt) - 1 + i]
            assert float(row.max() - row[tok]) < 0.1 * float(row.abs().max()), (i, tok)
    assert llm.runner.decode_graphs and llm.runner._graphs


def test_command_line_generates_from_a_robuvik_folder(tmp_path):
    import subprocess
    import sys
    d = _model_dir(tmp_path, "B")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "vllm_oxide_b200", "generate", d, "--prompt-ids", "5,9,2,44", "--max-new", "6", "--dtype", "float32",
                        "--max-model-len", "64", "--max-batch-tokens", "64", "--max-seqs", "2", "--num-pages", "16"],
                       cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    got = [int(x) for x in r.stdout.split()]
    toks = [5, 9, 2, 44]
    assert len(got) == 6
    logits = _plain_logits(d, toks + got)
    assert got[0] == int(logits[3].argmax())


def test_trace_program_replays_a_robuvik_folder(tmp_path):
    """bin/trace_run on a model folder: a prompt in two portions and two single tokens, logits of chosen places."""
    import subprocess
    import numpy as np
    d = _model_dir(tmp_path, "B")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    toks = _tokens(30, 131, 77)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:11], "want": [10]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[11:28], "want": [0, 16]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[28:29], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": toks[29:], "want": [0]}], "end": ["x"]}]
    out = os.path.join(str(tmp_path), "trace_out")
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out, "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900, cwd=root)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    want = _plain_logits(d, toks)
    assert not os.path.exists(os.path.join(out, "2.f32"))
    for step, places in ((0, [10]), (1, [11, 27]), (3, [29])):
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4").reshape(len(places), 131))
        assert _diff(got, want[places]) < TOL["float32"]
