"""The Fanopel configuration and its cache on the CPU: config.json's keys in and out, optional keys, what is refused, the
manifest of tensor names, a model folder with random weights; window groups of the cache manager that keep the first
tokens of a request; the plain model's mechanisms on examples worked out by hand."""
import json
import math
import os
import random

import pytest
import torch

from tests.plain import fanopel_plain as plain
from vllm_oxide_b200.config import FanopelConfig, KeyValueAttentionConfig, PlainExpertsConfig, architecture_for
from vllm_oxide_b200.csrc.build import runtime_module
from vllm_oxide_b200.errors import ConfigError
from vllm_oxide_b200 import models  # noqa: F401  (registers the architectures)

rt = runtime_module()


def _dict():
    moe = {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 6, "top": 2, "scale": 2.5, "groups": {"count": 3, "keep": 2}}}
    return {"architecture": "Fanopel", "vocab": 61, "width": 40, "max_positions": 96, "norm": {"eps": 1e-6}, "residual_mult": 0.3,
            "layers": [
                {"type": "attention", "mixer": {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 12, "scale": 0.3, "softcap": 5.0,
                                                "mask": {"size": 9, "keep_first": 4}}, "mlp": moe},
                {"type": "attention", "mixer": {"heads": 5, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.2,
                                                "mask": {"size": 30, "keep_first": 0}}, "mlp": None}]}


def test_keys_in_and_out_and_the_registry():
    d = _dict()
    cfg = FanopelConfig.from_dict(d)
    assert cfg.to_dict() == d
    assert FanopelConfig.from_dict(cfg.to_dict()) == cfg
    assert architecture_for(d).name == "Fanopel"
    assert cfg.layers[0].attention == KeyValueAttentionConfig(heads=6, kv_heads=3, dim=12, scale=0.3, softcap=5.0, window=9, keep_first=4)
    assert cfg.layers[0].mlp == PlainExpertsConfig(ff=20, experts=6, top=2, scale=2.5, groups=3, keep=2)
    assert cfg.layers[1].mlp is None and cfg.residual_mult == 0.3


def test_whole_numbers_are_taken_for_constants_and_optional_keys_switch_their_mechanism_off():
    d = _dict()
    d["residual_mult"] = 1
    d["layers"][0]["mixer"].update(softcap=7, scale=1)
    d["layers"][0]["mlp"]["router"]["scale"] = 2
    cfg = FanopelConfig.from_dict(d)
    assert (cfg.residual_mult, cfg.layers[0].attention.softcap, cfg.layers[0].mlp.scale) == (1.0, 7.0, 2.0)
    d["layers"][0]["mixer"].pop("mask")
    d["layers"][0]["mixer"].pop("softcap")
    d["layers"][0]["mixer"].pop("vdim")
    d["layers"][0]["mlp"]["router"].pop("groups")
    d["layers"][0]["mlp"]["router"].pop("scale")
    d.pop("residual_mult")
    cfg = FanopelConfig.from_dict(d)
    a = cfg.layers[0].attention
    assert (a.window, a.keep_first, a.softcap, cfg.layers[0].mlp.groups, cfg.layers[0].mlp.scale, cfg.residual_mult) == (0, 0, 0.0, 0, 1.0, 1.0)


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0].update(type="conv"), "type"),
    (lambda d: d["layers"][0]["mixer"].update(vdim=8), "vdim"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda d: d["layers"][0]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "choices"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=5), "choices"),
    (lambda d: d.pop("max_positions"), "max_positions"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_what_is_refused(change, word):
    d = json.loads(json.dumps(_dict()))
    change(d)
    with pytest.raises(ConfigError) as e:
        FanopelConfig.from_dict(d)
    assert word in str(e.value)


def test_manifest_names_and_a_model_folder(tmp_path):
    from vllm_oxide_b200.config.model_config import write_config_json
    from vllm_oxide_b200.models import fanopel_manifest
    from vllm_oxide_b200.weights import load_safetensors_weights, random_tensors
    from vllm_oxide_b200.weights.safetensors_io import write_safetensors
    cfg = FanopelConfig.from_dict(_dict())
    m = fanopel_manifest(cfg)
    assert m["pos"].shape == (96, 40) and m["l0.mix.q"].shape == (72, 40) and m["l0.mix.k"].shape == (36, 40)
    assert m["l0.mix.q.norm"].shape == (72,) and m["l0.mix.k.norm"].shape == (36,) and m["l0.mix.g"].shape == (6, 40)
    assert m["l0.mlp.e5.up"].shape == (20, 40) and m["l0.mlp.correction"].shape == (6,)
    assert "l0.mix.v" not in m and "l0.mlp.e0.gate" not in m and "l1.norm2" not in m and "l1.mlp.router" not in m
    assert cfg.param_count() == sum(int(torch.tensor(s.shape).prod()) for s in m.values())
    d = str(tmp_path)
    write_config_json(d, cfg.to_dict())
    write_safetensors(os.path.join(d, "model.safetensors"), random_tensors(m, 5, 0.1, torch.bfloat16, "cpu"))
    w = load_safetensors_weights(d, m, device="cpu")
    assert w.take("l1.mix.o").shape == (40, 80)


def test_slopes_of_head_counts_that_are_no_power_of_two():
    from vllm_oxide_b200.models.fanopel import distance_slopes
    assert distance_slopes(8).tolist() == [2.0 ** -(a + 1) for a in range(8)]
    assert distance_slopes(1).tolist() == [2.0 ** -8]
    assert torch.allclose(distance_slopes(6).double(), plain.slopes(6), rtol=1e-7)


# ------------------------------------------------------------------------------------ window groups that keep first tokens
@pytest.mark.parametrize("page,window,keep", [(4, 10, 3), (4, 10, 4), (4, 10, 9), (8, 3, 1), (4, 1, 6), (16, 20, 16)])
def test_kept_first_pages_stay_and_the_rest_behind_the_window_goes_back(page, window, keep):
    pages = 40
    c = rt.CacheManager(page, [rt.GroupSpec(rt.WINDOW, window, pages, keep)], 2)
    c.admit(1)
    rng = random.Random(window)
    length = 0
    first_table = None
    while length < 90:
        n = rng.randint(1, 7)
        assert c.reserve(1, n)
        table = c.block_table(1, 0)
        for p in range(length, length + n):            # every key that one of these queries reads lies in a page that is held
            for j in list(range(max(0, p + 1 - window), p + 1)) + list(range(min(keep, p + 1))):
                assert table[j // page] >= 0, (p, j)
        assert sum(x >= 0 for x in table) <= c.max_pages_held(0, 90) + -(-n // page)
        c.commit(1, n)
        length += n
        table = c.block_table(1, 0)
        kept = -(-keep // page)
        first_table = first_table if first_table is not None and len(first_table) == kept else table[:kept]
        assert table[:kept] == first_table[:len(table[:kept])]                   # the same pages all along
        dead = max(0, length + 1 - window) // page
        assert all(x == -1 for x in table[kept:dead]) and all(x >= 0 for x in table[max(kept, dead):])
        assert c.check_invariants() == ""
    c.release(1)
    assert c.num_free_pages(0) == pages and c.check_invariants() == ""


def test_kept_first_tokens_go_with_a_window():
    with pytest.raises(rt.RuntimeFault, match="kept first"):
        rt.CacheManager(4, [rt.GroupSpec(rt.FULL, 0, 4, 2)], 1)
    with pytest.raises(rt.RuntimeFault, match="kept first"):
        rt.CacheManager(4, [rt.GroupSpec(rt.WINDOW, 4, 4, -1)], 1)


def test_a_request_longer_than_the_pool_fits_through_its_window_and_kept_pages():
    # 6 pages of 4: a window of 9 holds at most 13 tokens' pages, kept first tokens one more page
    c = rt.CacheManager(4, [rt.GroupSpec(rt.WINDOW, 9, 6, 3)], 1)
    s = rt.Scheduler(c, 8, 1, 200, 4)
    assert c.max_pages_held(0, 150) == 5
    s.add_request(1, list(range(100)), rt.SamplingParams(max_new_tokens=20))
    done = 0
    while s.has_unfinished() and done < 400:
        plan = s.schedule()
        assert not plan.failed and plan.num_entries == 1
        s.update(plan, [7] * len(plan.sampling_ids()))
        done += 1
        assert c.check_invariants() == ""
    assert not s.has_unfinished()


# ------------------------------------------------------------------------------------ the plain model by hand
def test_visible_pairs():
    vis = plain.visible(7, 2, 3)
    want = [[j for j in range(i + 1) if i - j < 2 or j < 3] for i in range(7)]
    assert [[j for j in range(7) if vis[i, j]] for i in range(7)] == want
    assert plain.visible(5, None, 3).equal(torch.ones(5, 5).tril().bool())


def test_election_with_negative_choice_scores_and_groups_by_their_two_best():
    # sigmoid scores 0.5 everywhere; choice scores: group 0 {0.4, 0.4}, group 1 {0.6, -0.5}, group 2 {-1.5, -1.5}
    t = {"router": torch.zeros(6, 3, dtype=torch.float64),
         "correction": torch.tensor([-0.1, -0.1, 0.1, -1.0, -2.0, -2.0], dtype=torch.float64)}
    idx, w = plain.route(torch.ones(1, 3, dtype=torch.float64), t, "", {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}})
    assert sorted(idx[0].tolist()) == [0, 1] and torch.allclose(w, torch.full((1, 2), 1.5, dtype=torch.float64))
    idx, _ = plain.route(torch.ones(1, 3, dtype=torch.float64), t, "", {"experts": 6, "top": 4, "scale": 3.0, "groups": {"count": 3, "keep": 2}})
    assert sorted(idx[0].tolist()) == [0, 1, 2, 3]         # a negative choice score of a kept group beats "not standing"


def test_scores_are_capped_before_the_distance_is_taken_off():
    m = {"scale": 2.0, "softcap": 3.0}
    q, k = torch.ones(2, 1, 1, dtype=torch.float64) * 5, torch.ones(2, 1, 1, dtype=torch.float64) * 4
    s = plain.scores(q, k, m)
    assert math.isclose(float(s[0, 1, 0]), 3 * math.tanh(40 / 3) - 2.0 ** -8)
