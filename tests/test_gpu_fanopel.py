"""The Fanopel decoder in the engine against the plain implementation (tests/plain/fanopel_plain.py): small configurations
made here, random weights, float32 and bfloat16. Each mechanism alone (the kernels on inputs made so that a fault shows:
a key that stands out at the last kept first token, just behind it, at the window's first key and just outside, at a page's
border; choice scores below zero; groups whose best expert and whose two best disagree), models of one layer, whole
prompts against tokens one by one, portions down to two tokens, unequal requests side by side against each alone, pages
that are given back and used again, long decoding over windows, and greedy generation through `LLM`, the command line and
the trace program."""
import json
import os
import random

import pytest
import torch

from tests.plain import fanopel_plain as plain
from tests.util import max_rel_diff

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _configs():
    from vllm_oxide_b200.config import FanopelConfig as C, FanopelLayer as L, KeyValueAttentionConfig as AT, PlainExpertsConfig as FF
    att = AT(heads=4, kv_heads=2, dim=24, scale=0.25, softcap=6.0, window=11, keep_first=3)
    att_b = AT(heads=6, kv_heads=2, dim=16, scale=0.3, softcap=9.0, window=20, keep_first=9)                # kept tokens over a page's border
    att_odd = AT(heads=3, kv_heads=3, dim=10, scale=0.35, softcap=4.0, window=5, keep_first=1)              # sizes the tensor cores do not take
    att_nokeep = AT(heads=5, kv_heads=1, dim=32, scale=0.2, softcap=12.0, window=7)                         # nothing kept
    att_all = AT(heads=2, kv_heads=1, dim=8, scale=0.4, softcap=3.0)                                        # every earlier token
    att_one = AT(heads=1, kv_heads=1, dim=8, scale=0.4, window=1, keep_first=2)                             # itself and two kept tokens, no cap
    att_64 = AT(heads=8, kv_heads=2, dim=64, scale=0.1, softcap=8.0, window=40, keep_first=5)
    att_128 = AT(heads=3, kv_heads=1, dim=128, scale=0.09, softcap=15.0, window=70, keep_first=66)          # more kept tokens than a key tile holds
    att_96 = AT(heads=2, kv_heads=2, dim=96, scale=0.1, softcap=10.0, window=33, keep_first=2)
    moe = FF(ff=24, experts=6, top=2, scale=1.7, groups=3, keep=2)
    moe_flat = FF(ff=20, experts=5, top=3, scale=0.6)                                                       # no groups
    moe_ones = FF(ff=16, experts=4, top=1, scale=1.0, groups=4, keep=3)                                     # groups of one expert
    moe_one_group = FF(ff=12, experts=7, top=4, scale=2.0, groups=1, keep=1)
    return {
        "A": C(vocab=97, width=64, norm_eps=1e-5, max_positions=192, residual_mult=0.4, layers=(
            L(att, moe), L(att_b, moe_flat), L(att, None), L(att_nokeep, moe))),
        # a width that is no multiple of 4 or 8, other eps, a multiplier of 1, layers without feed-forward at both ends
        "B": C(vocab=131, width=42, norm_eps=1e-6, max_positions=160, residual_mult=1.0, layers=(
            L(att_odd, None), L(att_one, moe_ones), L(att_all, moe_one_group), L(att_odd, None))),
        # sizes of the tensor-core kernels
        "T": C(vocab=77, width=96, norm_eps=1e-5, max_positions=256, residual_mult=0.7, layers=(
            L(att_64, moe), L(att_128, moe_flat), L(att_96, None))),
        "attention": C(vocab=50, width=48, norm_eps=1e-5, max_positions=64, residual_mult=0.8, layers=(L(att, None),)),
        "moe": C(vocab=50, width=48, norm_eps=1e-5, max_positions=64, residual_mult=0.6, layers=(L(att_one, moe),)),
    }


def _model_dir(tmp_path, name, seed=11):
    """Random weights; queries, routers, gates and corrections are made large enough to matter."""
    from vllm_oxide_b200.config.model_config import write_config_json
    from vllm_oxide_b200.models import fanopel_manifest
    from vllm_oxide_b200.weights import random_tensors
    from vllm_oxide_b200.weights.safetensors_io import write_safetensors
    d = os.path.join(str(tmp_path), f"fanopel_{name}_{seed}")
    if os.path.exists(os.path.join(d, "model.safetensors")):
        return d
    cfg = _configs()[name]
    tensors = random_tensors(fanopel_manifest(cfg), seed, 0.25, torch.bfloat16, "cpu", norm_jitter=0.3)
    g = torch.Generator().manual_seed(seed)
    for n in list(tensors):
        if n.endswith(".router"):
            tensors[n] = (tensors[n].float() * 6).bfloat16()
        elif n.endswith(".correction"):
            tensors[n] = (torch.randn(tensors[n].shape, generator=g) * 0.5 - 0.6).bfloat16()      # choice scores on both sides of zero
        elif n.endswith(".mix.g"):
            tensors[n] = (tensors[n].float() * 2).bfloat16()
        elif n.endswith(".q.norm") or n.endswith(".k.norm"):
            tensors[n] = (tensors[n].float() * 2).bfloat16()
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
    bfloat16: the typical row tight (a router's close call may go to another expert than in float64, so single rows are
    judged in float32 only; a key that is skipped or a window one token off moves all later rows by far more)."""
    if dtype == "float32":
        rows = (got.double().cpu() - want).abs().amax(-1) / want.abs().max()
        return bool((rows < TOL[dtype] + 2 * getattr(want, "spread", 0.0)).all())
    err = _row_errors(got, want)
    return float(err.median()) < 4e-2 and float(err.quantile(0.7)) < 1e-1


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
def test_layer_norm_that_adds_a_multiple_first():
    from vllm_oxide_b200 import kernels
    torch.manual_seed(0)
    for h in (42, 64, 300, 1100, 2052, 4100, 9000):              # one to eight turns in registers, and rows in shared memory
        for dt in (torch.float32, torch.bfloat16):
            resid = torch.randn(5, h, device=DEV) * 3 + 0.5
            delta = (torch.randn(5, h, device=DEV) * 2 + 0.7).to(dt)
            w, b = torch.rand(h, device=DEV) + 0.5, torch.randn(h, device=DEV)
            for bias in (None, b):
                for mult in (1.0, -0.37):
                    r = resid.clone()
                    out = torch.empty(5, h, dtype=dt, device=DEV)
                    kernels.add_layernorm(r, delta, w, bias, 1e-5, out, mult=mult)
                    x = resid.double() + mult * delta.double()
                    want = plain.layer_norm(x, w.double(), 1e-5) + (bias.double() if bias is not None else 0)
                    assert _diff(r, x) < 1e-6
                    assert _diff(out, want) < (3e-6 if dt == torch.float32 else 6e-3)
            rows = _ints([4, 1])
            r = resid.clone()
            picked = torch.empty(2, h, dtype=dt, device=DEV)
            kernels.add_layernorm(r, delta, w, None, 1e-5, picked, rows, mult=0.25)          # looked at only: the residual stays
            assert torch.equal(r, resid)
            want = plain.layer_norm(resid.double() + 0.25 * delta.double(), w.double(), 1e-5)[[4, 1]]
            assert _diff(picked, want) < (3e-6 if dt == torch.float32 else 6e-3)
    # a row whose entries are large and nearly equal: the variance is the mean of the squared deviations
    r = 1000.0 + torch.randn(1, 64, device=DEV) * 0.01
    out = torch.empty(1, 64, device=DEV)
    kernels.add_layernorm(r, torch.zeros_like(r), torch.ones(64, device=DEV), None, 1e-5, out)
    assert _diff(out, plain.layer_norm(r.double(), torch.ones(64, dtype=torch.float64, device=DEV), 1e-5)) < 1e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,off", [(4, 2, 24, 0), (3, 3, 10, 5), (8, 2, 64, 16), (1, 1, 8, 0), (6, 2, 128, 8), (32, 8, 128, 0), (40, 8, 256, 8)])
def test_queries_and_keys_normed_as_a_whole(dtype, H, G, D, off):
    """q leaves with both norms' weights, k goes to its cache slot as projected and its 1 / rms beside it; padding rows and rows
    without a slot write nothing."""
    from vllm_oxide_b200 import kernels
    torch.manual_seed(D)
    T, page, pages, eps = 7, 8, 4, 1e-3
    proj = (torch.randn(T, off + (H + G) * D + 8, device=DEV) * torch.rand(T, 1, device=DEV) * 2).to(dtype)
    w = torch.randn(H * D, device=DEV)
    kc = torch.full((pages, G, page, D), float("nan"), dtype=dtype, device=DEV)
    ks = torch.full((pages, 1, page, 1), float("nan"), device=DEV)
    positions, slots = _ints([3, 4, 5, -1, 0, 1, 9]), _ints([17, 18, 0, -1, 31, -1, 8])
    q = torch.full((T, H * D), 7.0, dtype=dtype, device=DEV)
    kernels.whole_norm_prep(proj, off, positions, slots, w, eps, q, kc, ks, H, G, D)
    pq, pk = proj[:, off:off + H * D].double(), proj[:, off + H * D:off + (H + G) * D].double()
    want = plain.rms_norm(pq, w.double(), eps)
    live = [0, 1, 2, 4, 5, 6]
    assert _diff(q[live], want[live]) < (2e-6 if dtype == torch.float32 else 5e-3)
    assert bool((q[3] == 7.0).all())
    inv = 1.0 / torch.sqrt((pk * pk).mean(-1) + eps)
    written = torch.zeros(pages * page, dtype=torch.bool)
    for r, slot in ((0, 17), (1, 18), (2, 0), (4, 31), (6, 8)):
        assert torch.equal(kc[slot // page, :, slot % page].reshape(-1), proj[r, off + H * D:off + (H + G) * D])
        assert abs(float(ks[slot // page, 0, slot % page, 0]) / float(inv[r]) - 1) < 1e-6
        written[slot] = True
    assert torch.isnan(ks.view(-1).cpu()).equal(~written)
    assert torch.isnan(kc[:, 0, :, 0].reshape(-1).cpu()).equal(~written)


# ------------------------------------------------------------------------------------ attention kernels
def _paged(total, page, heads_widths, dtypes, spare=3):
    """Block tables over scattered pages for requests of `total` tokens; cache tensors full of NaN."""
    pages_per = [-(-t // page) for t in total]
    n = sum(pages_per) + spare
    perm = torch.randperm(n)
    tables = torch.full((len(total), max(pages_per) + 2), -1, dtype=torch.int32)
    at = 0
    for s, pp in enumerate(pages_per):
        tables[s, :pp] = perm[at:at + pp].to(torch.int32)
        at += pp
    caches = [torch.full((n, h, page, w), float("nan"), dtype=dt, device=DEV) for (h, w), dt in zip(heads_widths, dtypes)]
    return tables, caches


def _fill(cache, tables, s, x, page, idx):
    """The tokens `idx` of x [tokens, heads, width] of request s into its pages."""
    idx = torch.tensor(idx)
    pg, off = tables[s, idx // page].long(), idx % page
    cache[pg.to(DEV), :, off.to(DEV)] = x[idx].to(device=DEV, dtype=cache.dtype)


def _attention_plain(q, k, v, first_pos, window, keep, scale, cap, slopes, gate):
    """q [n, H, D] at positions first_pos ..; k, v [total, G, .]: the rows' results [n, H * DV] and weights [H, n, total]."""
    n, H, _ = q.shape
    total, G, _ = k.shape
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    i, j = torch.arange(first_pos, first_pos + n)[:, None], torch.arange(total)[None, :]
    if slopes is not None:
        s = s - slopes[:, None, None] * (i - j).double()
    vis = j <= i
    if window:
        vis = vis & ((i - j < window) | (j < keep))
    w = torch.softmax(s.masked_fill(~vis, float("-inf")), dim=-1)
    o = torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(H // G, 1)) * torch.sigmoid(gate)[:, :, None]
    return o.reshape(n, -1), w


CASES = [(4, 2, 24, 24, 21, 5, 6.0, True), (3, 3, 10, 6, 9, 3, 5.0, True), (8, 4, 64, 64, 48, 6, 8.0, True), (6, 2, 128, 128, 100, 70, 20.0, True),
         (2, 1, 96, 96, 70, 130, 0.0, True), (2, 2, 16, 16, 7, 0, 4.0, True), (1, 1, 8, 8, 1, 1, 2.0, True), (5, 1, 64, 64, 130, 9, 9.0, True),
         (16, 1, 64, 64, 90, 64, 30.0, False), (4, 4, 32, 48, 64, 3, 3.0, True), (4, 2, 128, 128, 0, 0, 10.0, True), (2, 1, 64, 64, 33, 65, 12.0, True)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shared", [True, False])
@pytest.mark.parametrize("H,G,D,DV,window,keep,cap,bias", CASES)
def test_window_with_kept_first_tokens_linear_bias_and_values_that_are_keys(dtype, shared, H, G, D, DV, window, keep, cap, bias):
    """Two requests in one batch over scattered pages: a portion of rows behind a context that is in the cache and a single
    decoded token far into its context. One row looks at the last kept first token, the decoded one at the first key of its
    window; the token just behind the kept ones and the one just outside the window would outweigh everything if they were
    seen. Everything that no row may read holds NaN. `shared`: the values are the keys as cached, each with a number of its own
    that its scores are multiplied by; else keys and values apart."""
    from vllm_oxide_b200 import kernels
    if shared and D != DV:
        pytest.skip("the values are the keys")
    torch.manual_seed(3)
    page, scale = 8, 0.3
    ctxs, lens = (150, 320), (70, 1)
    total = [c + n for c, n in zip(ctxs, lens)]
    tables, (kc, vc, ks) = _paged(total, page, [(G, D), (G, DV), (1, 1)], [dtype, dtype, torch.float32])
    k = [torch.randn(t, G, D) * 0.5 for t in total]
    v = [torch.randn(t, G, DV) for t in total]
    inv = [torch.rand(t, 1, 1) + 0.5 for t in total] if shared else [torch.ones(t, 1, 1) for t in total]
    T, group, far_row = sum(lens), H // G, 60                     # request 0, position 210
    q = torch.randn(T, H, D) * 0.5
    slopes = torch.rand(H) * 0.02 if bias else None

    def aim(row, s, key, weight):
        for a in range(H):
            kk = (k[s] * inv[s])[key, a // group]
            q[row, a] = weight * kk / kk.norm() ** 2 / scale
    pos = (ctxs[0] + far_row, total[1] - 1)
    lo = [max(0, p + 1 - window) if window else 0 for p in pos]
    aim(far_row, 0, keep - 1 if keep else lo[0], 14.0)
    aim(T - 1, 1, lo[1] if window else 5, 14.0)
    if window:      # what must not be seen: just behind the kept tokens, just outside the window
        for s, row in ((0, far_row), (1, T - 1)):
            for key in (keep, lo[s] - 1):
                if keep <= key < lo[s]:
                    k[s][key] = 40.0 * q[row, 0] / q[row, 0].norm() ** 2 / scale
    readable = []
    for s in range(2):
        first = max(0, ctxs[s] + 1 - window) if window else 0
        readable.append(sorted(set(range(min(keep, total[s]))) | set(range(first, total[s]))))
        _fill(kc, tables, s, k[s], page, readable[s])
        _fill(vc, tables, s, v[s], page, readable[s])
        _fill(ks, tables, s, inv[s], page, readable[s])
        for lp in range(tables.shape[1]):                         # pages that hold nothing readable have been given back
            if not any(j // page == lp for j in readable[s]):
                tables[s, lp] = -1
    positions = torch.cat([torch.arange(ctxs[s], total[s]) for s in range(2)]).to(device=DEV, dtype=torch.int32)
    row_seq = torch.cat([torch.full((lens[s],), s) for s in range(2)]).to(device=DEV, dtype=torch.int32)
    qd = q.reshape(T, H * D).to(device=DEV, dtype=dtype)
    wide_gate = torch.randn(T, H + 3).to(device=DEV, dtype=dtype)
    gd = wide_gate[:, 3:]
    sd = slopes.to(DEV) if bias else None
    kw = dict(chunk=0, softcap=cap, dist_bias=None, keep_first=keep, dist_slopes=sd, key_scale=ks if shared else None)
    vals = kc if shared else vc
    outs = {}
    wide = torch.full((T, H * DV + 8), float("nan"), dtype=dtype, device=DEV)
    kernels.flex_attention(qd, wide[:, 8:], kc, vals, tables.to(DEV), row_seq, positions, H, G, D, DV, scale, window, None, gd, 1.0, **kw)
    outs["general"] = wide[:, 8:]
    if dtype == torch.bfloat16 and kernels.attn_prefill_mma_any_supported(H, G, D, DV, page) and (shared or not (keep or bias)):
        wide2 = torch.full((T, H * DV + 8), float("nan"), dtype=dtype, device=DEV)
        kernels.attn_prefill_mma_any(qd, wide2[:, 8:], kc, vals, tables.to(DEV), _ints([0, lens[0], T]), _ints(ctxs), 2, max(lens), H, G, D, DV,
                                     scale, window, None, gd, 1.0, **kw)
        assert bool(torch.isnan(wide2[:, :8]).all())
        outs["portions"] = wide2[:, 8:]
    decode = {}
    if dtype == torch.bfloat16 and D == DV and D in (64, 128) and (shared or not (keep or bias)):
        last = torch.tensor([lens[0] - 1, T - 1], device=DEV)
        for splits in (1, 2, 3, 8, 20):
            o2 = torch.full((2, H * DV), float("nan"), dtype=dtype, device=DEV)
            part = torch.empty(kernels.attn_decode_partial_floats(2, G, D, splits), device=DEV) if splits > 8 else None
            arrived = torch.zeros(2 * G, dtype=torch.int32, device=DEV) if splits > 8 else None
            kernels.attn_decode_mma(qd[last].contiguous(), o2, kc, vals, tables.to(DEV), positions[last].contiguous(), H, G, D, scale, window,
                                    splits, part, arrived, None, gd[last], 1.0, **kw)
            decode[splits] = o2
            assert arrived is None or int(arrived.abs().max()) == 0
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    r0 = 0
    for s in range(2):
        keys, vv = (k[s].to(dtype).double() * inv[s].double()), (k[s] if shared else v[s]).to(dtype).double()
        qq = qd[r0:r0 + lens[s]].cpu().double().reshape(lens[s], H, D)
        want, w = _attention_plain(qq, keys, vv, ctxs[s], window, keep, scale, cap, slopes.double() if bias else None,
                                   gd[r0:r0 + lens[s]].cpu().double())
        for name, out in outs.items():
            got = out[r0:r0 + lens[s]].cpu()
            assert not bool(torch.isnan(got).any()), (name, s)
            assert max_rel_diff(got, want) < tol, (name, s)
        for splits, o2 in decode.items():
            assert max_rel_diff(o2[s:s + 1].cpu(), want[-1:]) < tol, (splits, s)
        if window and keep and s == 0 and keep + window < pos[0] and not cap and not bias:
            assert float(w[0, far_row, keep - 1]) > 0.5           # the far key is what the row is made of
        r0 += lens[s]
    assert bool(torch.isnan(wide[:, :8]).all())


def test_what_the_kernels_refuse():
    from vllm_oxide_b200 import kernels
    from vllm_oxide_b200.errors import ShapeError
    tables, (kc, vc, ks) = _paged([20], 8, [(1, 64), (1, 64), (1, 1)], [torch.bfloat16, torch.bfloat16, torch.float32])
    q, out = torch.zeros(1, 64, dtype=torch.bfloat16, device=DEV), torch.zeros(1, 64, dtype=torch.bfloat16, device=DEV)
    a = (tables.to(DEV), _ints([0]), _ints([5]), 1, 1, 64, 64, 0.1)
    with pytest.raises(ShapeError, match="kept first"):
        kernels.flex_attention(q, out, kc, vc, *a, keep_first=3)
    with pytest.raises(ShapeError, match="both"):
        kernels.flex_attention(q, out, kc, vc, *a, dist_slopes=torch.ones(1, device=DEV), dist_bias=(torch.ones(1, device=DEV),) * 2)
    with pytest.raises(ShapeError, match="float32 per cached token"):
        kernels.flex_attention(q, out, kc, kc, *a, key_scale=ks[:, :, :4])
    with pytest.raises(ShapeError, match="values that are the cached keys"):
        kernels.attn_decode_mma(q, out, kc, vc, tables.to(DEV), _ints([5]), 1, 1, 64, 0.1, 4, key_scale=ks)
    with pytest.raises(ShapeError, match="gate must be"):
        kernels.flex_attention(q, out, kc, vc, *a, gate=torch.zeros(1, 2, dtype=torch.bfloat16, device=DEV))


def _step_ctx(positions, starts, tables, slot_map, dtype, max_new, decode_only, ctx_len=0):
    from vllm_oxide_b200.parts.base import StepContext, Workspace
    n, s = len(positions), len(starts) - 1
    return StepContext(rows=n, seqs=s, dtype=dtype, tokens=_ints([0] * n), positions=_ints(positions), row_seq=_ints([0] * n),
                       seq_starts=_ints(starts), context_lens=_ints([ctx_len] * s), seq_lens=_ints([0] * s), state_slots=_ints([0] * s),
                       logit_rows=_ints([0]), slot_mapping=[_ints(slot_map)] if slot_map is not None else [],
                       block_tables=[tables.to(DEV)] if tables is not None else [], workspace=Workspace(64 << 20, DEV),
                       max_new=max_new, decode_only=decode_only)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,window,keep,cap", [(4, 2, 24, 13, 4, 5.0), (2, 2, 10, 6, 0, 3.0), (8, 2, 64, 30, 7, 8.0), (3, 1, 128, 65, 3, 0.0)])
def test_the_mixer_whole_in_portions_and_token_by_token(dtype, H, G, D, window, keep, cap):
    """One request of 90 tokens through the mixer: whole, in portions, token by token, against the plain attention; one token
    just outside the window of row 80 is much like row 80's own."""
    from vllm_oxide_b200.models.fanopel import distance_slopes
    from vllm_oxide_b200.parts.base import LayerCache
    from vllm_oxide_b200.parts.flex_attention import SoftmaxAttention
    torch.manual_seed(H + D)
    width, T, page = 40, 90, 8
    t = {"q": torch.randn(H * D, width) * 0.3, "k": torch.randn(G * D, width) * 0.3, "q.norm": torch.rand(H * D) * 2 + 0.5,
         "k.norm": torch.rand(G * D) * 2 + 0.5, "g": torch.randn(H, width) * 0.5, "o": torch.randn(width, H * D) * 0.2}
    t = {n: x.bfloat16() for n, x in t.items()}
    mixer = SoftmaxAttention(t["q"], t["k"], None, t["o"], H, G, D, D, 0.2, window=window, keep_first=keep, softcap=cap,
                             dist_slopes=distance_slopes(H), values_are_keys=True, q_pre_norm=t["q.norm"], k_pre_norm=t["k.norm"],
                             pre_norm_eps=1e-5, gate_weight=t["g"], gate_per_head=True, dtype=dtype, device=DEV)
    assert mixer.cache_spec().keep_first == keep and mixer.w_in.shape[0] % 8 == 0
    x = torch.randn(T, width)
    x[80 - window] = x[80]
    x = x.to(dtype)
    m = {"heads": H, "kv_heads": G, "dim": D, "scale": 0.2, "softcap": cap, "mask": {"size": window, "keep_first": keep}}
    want = plain.attention(x.double(), {n: v.double() for n, v in t.items()}, "", m, 1e-5)
    for cuts in ([T], [5, 2, 43, 1, 39], [60] + [1] * 30):
        tables, caches = _paged([T], page, [(G, D), (1, 1)], [dtype, torch.float32])
        cache = LayerCache(tensors=tuple(caches), group=0, write=True)
        got, at = [], 0
        for n in cuts:
            pos = list(range(at, at + n))
            slot_map = [int(tables[0, p // page]) * page + p % page for p in pos]
            ctx = _step_ctx(pos, [0, n], tables, slot_map, dtype, n, n == 1, at)
            got.append(mixer.forward(x[at:at + n].to(DEV), ctx, cache, None).clone())
            assert ctx.workspace.high_water <= mixer.workspace_bytes(n) + 256 * 8 + n * width * 4
            at += n
        assert _diff(torch.cat(got), want) < (2e-5 if dtype == torch.float32 else 3e-2), cuts


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,DV,keep,slopes", [(4, 2, 64, 64, 5, True), (2, 2, 24, 40, 3, False), (2, 1, 128, 128, 0, True)])
def test_kept_first_tokens_and_the_linear_bias_with_values_of_their_own(dtype, H, G, D, DV, keep, slopes):
    """The same options in a mixer that has value projections and no norms (any of the kernels may take it)."""
    from vllm_oxide_b200.parts.base import LayerCache
    from vllm_oxide_b200.parts.flex_attention import SoftmaxAttention
    torch.manual_seed(D)
    width, T, page, window = 40, 70, 8, 17
    w = {n: (torch.randn(r, width) * 0.3).bfloat16() for n, r in (("q", H * D), ("k", G * D), ("v", G * DV))}
    wo, sl = (torch.randn(width, H * DV) * 0.2).bfloat16(), torch.rand(H) * 0.1
    mixer = SoftmaxAttention(w["q"], w["k"], w["v"], wo, H, G, D, DV, 0.1, window=window, keep_first=keep, softcap=6.0,
                             dist_slopes=sl if slopes else None, dtype=dtype, device=DEV)
    x = torch.randn(T, width).to(dtype)
    q, k, v = ((x.double() @ w[n].double().T).reshape(T, -1, z) for n, z in (("q", D), ("k", D), ("v", DV)))
    want, _ = _attention_plain(q, k, v, 0, window, keep, 0.1, 6.0, sl.double() if slopes else None, torch.full((T, H), 50.0, dtype=torch.float64))
    want = want @ wo.double().T
    for cuts in ([T], [9, 2, 40] + [1] * 19):
        tables, caches = _paged([T], page, [(G, D), (G, DV)], [dtype, dtype])
        cache = LayerCache(tensors=tuple(caches), group=0, write=True)
        got, at = [], 0
        for n in cuts:
            pos = list(range(at, at + n))
            ctx = _step_ctx(pos, [0, n], tables, [int(tables[0, p // page]) * page + p % page for p in pos], dtype, n, n == 1, at)
            got.append(mixer.forward(x[at:at + n].to(DEV), ctx, cache, None).clone())
            at += n
        assert _diff(torch.cat(got), want) < (2e-5 if dtype == torch.float32 else 3e-2), cuts


# ------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("E,top,groups,keep,shift", [(6, 2, 3, 2, -0.7), (10, 3, 2, 1, 0.0), (5, 3, 0, 0, -0.5), (4, 1, 4, 3, -2.0), (7, 4, 1, 1, 0.4),
                                                      (40, 8, 8, 3, -1.0), (64, 6, 16, 5, -1.8)])
def test_election_by_sigmoid_scores_with_a_correction(E, top, groups, keep, shift):
    """Choice scores on both sides of zero; groups scored by their two best experts; the weights are made of the scores without
    the correction."""
    from vllm_oxide_b200 import kernels
    torch.manual_seed(E + top)
    T, width = 203, 44
    router = torch.randn(E, width)
    corr = torch.randn(E) * 0.6 + shift
    x = torch.randn(T, width)
    r = {"experts": E, "top": top, "scale": 1.9}
    if groups:
        r["groups"] = {"count": groups, "keep": keep}
    t = {"router": router.double(), "correction": corr.double()}
    want_idx, want_w = plain.route(x.double(), t, "", r)
    low_idx, _ = plain.route(x, {"router": router, "correction": corr}, "", r)
    clear = (want_idx.sort(-1).values == low_idx.sort(-1).values).all(-1)                # no close call
    assert float(clear.double().mean()) > 0.97
    positions = torch.arange(T, dtype=torch.int32, device=DEV)
    positions[5] = -1
    idx, w = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    kernels.moe_route(x.to(DEV), router.to(DEV), positions, top, groups, keep, True, idx, w, score="sigmoid", correction=corr.to(DEV),
                      group_best=2, eps=1e-20, out_scale=1.9)
    assert bool((idx[5] == -1).all()) and bool((w[5] == 0).all())
    clear[5] = False
    got = torch.zeros(T, E, dtype=torch.float64)
    ok = idx.cpu() >= 0
    assert bool(ok[clear].all())
    got.scatter_(1, idx.cpu().clamp(min=0).long(), w.cpu().double() * ok)
    want = torch.zeros(T, E, dtype=torch.float64).scatter_(1, want_idx, want_w)
    assert _diff(got[clear], want[clear]) < 3e-6
    if groups > 1 and E // groups > 1 and keep < groups:                                  # scored by the best alone it would go elsewhere
        s = torch.sigmoid(x.double() @ router.double().T) + corr.double()
        best1 = s.view(T, groups, -1).amax(-1).topk(keep, -1).indices.sort(-1).values
        best2 = s.view(T, groups, -1).topk(2, -1).values.sum(-1).topk(keep, -1).indices.sort(-1).values
        assert bool((best1 != best2).any())
    if shift < 0:                                                                         # a choice score below zero was chosen somewhere
        s = torch.sigmoid(x.double() @ router.double().T) + corr.double()
        assert bool((s.gather(1, want_idx) < 0).any())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,width,ff,E,top,groups,keep", [(9, 48, 24, 6, 2, 3, 2), (70, 42, 20, 5, 1, 0, 0), (33, 64, 136, 5, 3, 0, 0), (600, 64, 32, 4, 2, 2, 1),
                                                          (700, 72, 200, 4, 3, 4, 3)])
def test_experts_without_a_gate(dtype, T, width, ff, E, top, groups, keep):
    """The routed feed-forward against every chosen expert done plainly: small tiles, large tiles, sizes that 16-byte copies do
    not take, hidden sizes that end inside a tile."""
    from vllm_oxide_b200.parts.moe import RoutedExperts
    torch.manual_seed(T)
    t = {"router": torch.randn(E, width) * 3, "correction": torch.randn(E) * 0.3}
    for e in range(E):
        t[f"e{e}.up"], t[f"e{e}.down"] = torch.randn(ff, width) * 0.3, torch.randn(width, ff) * 0.3
    t = {k: v.bfloat16() for k, v in t.items()}
    part = RoutedExperts(t["router"], None, [t[f"e{e}.up"] for e in range(E)], [t[f"e{e}.down"] for e in range(E)], top, groups, keep,
                         renormalize=True, dtype=dtype, device=DEV, activation="relu2", score="sigmoid", correction=t["correction"], group_best=2,
                         renorm_eps=1e-20, weight_scale=0.7)
    x = torch.randn(T, width).to(dtype)
    r = {"experts": E, "top": top, "scale": 0.7}
    if groups:
        r["groups"] = {"count": groups, "keep": keep}
    want = plain.moe_ff(x.double(), {k: v.double() for k, v in t.items()}, "", {"router": r})
    ctx = _step_ctx(list(range(T)), [0, T], None, None, dtype, T, False)
    got = part.forward(x.to(DEV), ctx)
    assert ctx.workspace.high_water <= part.workspace_bytes(T)
    err = _row_errors(got, want)
    if dtype == torch.float32:
        assert float(err.quantile(0.98)) < 2e-6 and float(err.median()) < 1e-6           # a close call may go either way
    else:
        assert float(err.median()) < 2e-2 and float(err.quantile(0.9)) < 6e-2


# ------------------------------------------------------------------------------------ models in the engine
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["attention", "moe"])
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
        assert _diff(single, whole) < 3e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "T"])
def test_portions_unequal_batches_and_reuse(tmp_path, name, dtype):
    """Four requests of unequal length in a pool that cannot hold them all at once: portions from 2 tokens up beside single
    tokens, portions that end inside a page, a window and the kept first tokens, a request that sits out a step, a fourth
    request that takes over a slot and pages that were given back in the middle. Every row equals the plain model's."""
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
            assert _diff(alone, got[k]) < 5e-6, k
        else:
            err = _row_errors(got[k], alone)
            assert float(err.median()) < 1.5e-2 and float(err.quantile(0.9)) < 6e-2, (k, float(err.median()), float(err.quantile(0.9)))


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


def test_the_stream_after_every_layer(tmp_path):
    """Layer by layer in float32: the residual with what is still pending (times the multiplier) equals the plain model's."""
    from vllm_oxide_b200.replay.trace import TraceSession
    for name in ("A", "B"):
        d = _model_dir(tmp_path, name)
        toks = _tokens(50, _configs()[name].vocab, 8)
        layers = []
        _plain_logits(d, toks, layers)
        runner = _runner(d, "float32")
        mult = _configs()[name].residual_mult
        seen = []
        runner.after_block = lambda i, resid, pending: seen.append((resid + mult * pending)[:len(toks)].clone())
        _replay(TraceSession(runner), {"a": toks}, [[("a", len(toks))]])
        assert len(seen) == len(layers)
        for i, got in enumerate(seen):
            assert _diff(got.cpu(), layers[i]) < 1e-5, (name, i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "T"])
def test_long_decoding_over_page_borders_and_windows(tmp_path, name, dtype):
    """150 tokens, all but six of them one by one: windows of 7 to 70 pass over decoded tokens, the window groups give their
    pages back on the way and keep those of the first tokens."""
    from vllm_oxide_b200.replay.trace import TraceSession
    d = _model_dir(tmp_path, name)
    toks = _tokens(150, _configs()[name].vocab, 9)
    want = _plain_logits(d, toks)
    runner = _runner(d, dtype, page=8, pages=20, max_seqs=2)
    _poison(runner)
    s = TraceSession(runner)
    got = _replay(s, {"a": toks + [0]}, [[("a", 6)]] + [[("a", 1)]] * 144)["a"]
    assert _close(got, want, dtype)
    free = [runner.manager.num_free_pages(g) for g in range(runner.pools.num_groups)]
    assert all(f > 0 for f in free), free                          # pages behind the windows went back while the request lives


def test_a_window_one_token_off_or_a_mechanism_left_out_would_show(tmp_path):
    """The plain model with every window one token longer, one kept token more or fewer, without the cap, the gate, the
    correction, the groups or a constant differs from itself by far more than the tolerance: the tests above can tell."""
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

    def mask(key, by):
        def change(c, t):
            for x in c["layers"]:
                x["mixer"]["mask"][key] = max(0, x["mixer"]["mask"].get(key, 0) + by)
        return change

    def no_cap(c, t):
        for x in c["layers"]:
            x["mixer"].pop("softcap", None)

    def no_groups(c, t):
        for x in c["layers"]:
            (x["mlp"] or {}).get("router", {}).pop("groups", None)

    def zero(suffix):
        def change(c, t):
            for n in t:
                if n.endswith(suffix):
                    t[n] = torch.zeros_like(t[n])
        return change

    def ones(suffix):
        def change(c, t):
            for n in t:
                if n.endswith(suffix):
                    t[n] = torch.ones_like(t[n])
        return change

    def mult(c, t):
        c["residual_mult"] = 1.0
    for change in (mask("size", 1), mask("size", -1), mask("keep_first", 1), mask("keep_first", -1), mask("keep_first", -99), no_cap, no_groups,
                   zero(".mix.g"), zero(".correction"), zero("pos"), ones(".q.norm"), ones(".k.norm"), mult):
        assert _diff(run(change), want) > 1e-3, getattr(change, "__name__", change)


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler(tmp_path, graphs):
    """More requests than state slots and a pool that forces preemption and recomputation: every generated token is the
    plain model's argmax given what came before. With CUDA graphs the decode steps are recorded and replayed."""
    from vllm_oxide_b200.config import EngineConfig
    from vllm_oxide_b200.engine import LLM, ModelRunner
    from vllm_oxide_b200.sampling import SamplingParams
    d = _model_dir(tmp_path, "A")
    eng = EngineConfig(max_batch_tokens=64, max_seqs=3, max_model_len=64, block_size=8, num_pages=9, dtype="float32", cuda_graphs=graphs)
    llm = LLM(ModelRunner.from_dir(d, eng))
    prompts = [_tokens(n, 97, 20 + n) for n in (14, 9, 17, 5, 2)]
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
            assert float(row.max() - row[tok]) < 0.08 * float(row.abs().max()), (i, tok)
    assert llm.runner.decode_graphs and llm.runner._graphs


def test_positions_beyond_the_learned_table_are_refused(tmp_path):
    from vllm_oxide_b200.replay.trace import TraceSession
    d = _model_dir(tmp_path, "attention")
    runner = _runner(d, "float32")
    assert runner.max_model_len == 64
    s = TraceSession(runner)
    _replay(s, {"a": _tokens(64, 50, 1)}, [[("a", 64)]])
    with pytest.raises(s.rt.RuntimeFault, match="block table"):
        _replay(s, {"b": _tokens(65, 50, 1)}, [[("b", 65)]], first_step=5)


def test_command_line_generates_from_a_fanopel_folder(tmp_path):
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


def test_trace_program_replays_a_fanopel_folder(tmp_path):
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
