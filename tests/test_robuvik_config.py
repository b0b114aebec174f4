"""The Robuvik configuration on the CPU: config.json's keys in and out, optional keys, what is refused, the manifest of tensor
names, a model folder with random weights, the order in which layers and passes run, stretched rotary frequencies; the plain
model's mechanisms on examples worked out by hand."""
import json
import math
import os

import pytest
import torch

from tests.plain import robuvik_plain as plain
from vllm_oxide_b200.config import (BigramConfig, DenseOrExpertsConfig, GatedLatentConfig, RobuvikConfig, StretchedRotaryConfig,
                                    WindowAttentionConfig, architecture_for)
from vllm_oxide_b200.errors import ConfigError
from vllm_oxide_b200 import models  # noqa: F401  (registers the architectures)


def _dict():
    sc = {"factor": 3.0, "original": 90.0, "fast": 9.0, "slow": 2.0}
    att = {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 10, "scale": 0.3, "mask": {"size": 9}, "rot": {"dims": 8, "base": 300.0, "scaling": sc}}
    lat = {"heads": 5, "dim": 7, "rot_dim": 6, "vdim": 9, "kv_rank": 14, "q_rank": 11, "scale": 0.2, "rot": {"dims": 6, "base": 150.0, "scaling": sc}}
    moe = {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 6, "top": 2}, "shared": {"ff": 13}}
    return {"architecture": "Robuvik", "vocab": 61, "width": 40, "norm": {"eps": 1e-6},
            "embedding": {"bigram": {"buckets": 23, "mul_prev": 7, "mul_cur": 5}}, "loop": {"start": 0, "stop": 2, "times": 3},
            "layers": [{"type": "attention", "mixer": att, "mlp": moe}, {"type": "latent_attention", "mixer": lat, "mlp": None},
                       {"type": "latent_attention", "mixer": lat, "mlp": {"kind": "dense", "ff": 33}}]}


def test_keys_in_and_out_and_the_registry():
    d = _dict()
    cfg = RobuvikConfig.from_dict(d)
    assert cfg.to_dict() == d
    assert RobuvikConfig.from_dict(cfg.to_dict()) == cfg
    assert architecture_for(d).name == "Robuvik"
    rot = StretchedRotaryConfig(dims=8, base=300.0, factor=3.0, original=90.0, fast=9.0, slow=2.0)
    assert cfg.layers[0].attention == WindowAttentionConfig(heads=6, kv_heads=3, dim=12, vdim=10, scale=0.3, rot=rot, window=9)
    assert cfg.layers[0].mlp == DenseOrExpertsConfig("moe", ff=20, experts=6, top=2, shared_ff=13)
    assert cfg.layers[1].latent == GatedLatentConfig(heads=5, dim=7, rot_dim=6, vdim=9, kv_rank=14, q_rank=11, scale=0.2,
                                                     rot=StretchedRotaryConfig(dims=6, base=150.0, factor=3.0, original=90.0, fast=9.0, slow=2.0))
    assert cfg.layers[1].mlp is None and cfg.layers[2].mlp == DenseOrExpertsConfig("dense", ff=33)
    assert cfg.bigram == BigramConfig(23, 7, 5) and cfg.loop == (0, 2, 3)


def test_whole_numbers_are_taken_for_constants_and_optional_keys_switch_their_mechanism_off():
    d = _dict()
    d["layers"][0]["mixer"]["scale"] = 1
    d["layers"][0]["mixer"]["rot"]["base"] = 300
    d["layers"][0]["mixer"]["rot"]["scaling"].update(factor=3, original=90, fast=9, slow=2)
    assert RobuvikConfig.from_dict(d).layers[0].attention.rot == RobuvikConfig.from_dict(_dict()).layers[0].attention.rot
    d["layers"][0]["mixer"].pop("mask")
    d["layers"][0]["mixer"].pop("rot")
    d["layers"][0]["mlp"].pop("shared")
    d["layers"][1]["mixer"]["rot"].pop("dims")
    d["layers"][1]["mixer"]["rot"].pop("scaling")
    d.pop("embedding")
    d.pop("loop")
    cfg = RobuvikConfig.from_dict(d)
    assert (cfg.layers[0].attention.window, cfg.layers[0].attention.rot, cfg.layers[0].mlp.shared_ff) == (0, None, 0)
    assert cfg.layers[1].latent.rot == StretchedRotaryConfig(dims=6, base=150.0)
    assert cfg.bigram is None and cfg.loop is None and [i for i, _ in cfg.run_order()] == [0, 1, 2]
    m = models.robuvik_manifest(cfg)
    assert "bigram" not in m and "loop.step" not in m and "l0.mlp.shared.up" not in m


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0].update(type="conv"), "type"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "rotated"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=14), "rotated"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "factor"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=4), "rot_dim"),
    (lambda d: d["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][0]["mlp"].update(kind="other"), "kind"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "choices"),
    (lambda d: d["layers"][0]["mlp"]["shared"].update(ff=0), "ff"),
    (lambda d: d["loop"].update(stop=4), "loop"),
    (lambda d: d["loop"].update(times=0), "loop"),
    (lambda d: d["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda d: d["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_what_is_refused(change, word):
    d = json.loads(json.dumps(_dict()))
    change(d)
    with pytest.raises(ConfigError) as e:
        RobuvikConfig.from_dict(d)
    assert word in str(e.value)


def test_manifest_names_and_a_model_folder(tmp_path):
    from vllm_oxide_b200.config.model_config import write_config_json
    from vllm_oxide_b200.weights import load_safetensors_weights, random_tensors
    from vllm_oxide_b200.weights.safetensors_io import write_safetensors
    cfg = RobuvikConfig.from_dict(_dict())
    m = models.robuvik_manifest(cfg)
    assert m["bigram"].shape == (24, 40) and m["loop.step"].shape == (3, 40)
    assert m["l0.mix.q"].shape == (72, 40) and m["l0.mix.k.b"].shape == (36,) and m["l0.mix.v"].shape == (30, 40) and m["l0.mix.o"].shape == (40, 60)
    assert m["l1.mix.dq"].shape == (11, 40) and m["l1.mix.uq"].shape == (65, 11) and m["l1.mix.dkv"].shape == (20, 40)
    assert m["l1.mix.uk"].shape == (35, 14) and m["l1.mix.uv"].shape == (45, 14) and m["l1.mix.g"].shape == (45, 40)
    assert m["l0.mlp.e5.gate"].shape == (20, 40) and m["l0.mlp.shared.down"].shape == (40, 13) and m["l2.mlp.up"].shape == (33, 40)
    assert "l1.mlp.up" not in m and "l0.norm2" not in m and "l2.mlp.gate" not in m
    assert cfg.param_count() == sum(int(torch.tensor(s.shape).prod()) for s in m.values())
    d = str(tmp_path)
    write_config_json(d, cfg.to_dict())
    write_safetensors(os.path.join(d, "model.safetensors"), random_tensors(m, 5, 0.1, torch.bfloat16, "cpu"))
    assert load_safetensors_weights(d, m, device="cpu").take("l1.mix.o").shape == (40, 45)


@pytest.mark.parametrize("loop,want", [
    (None, [(0, None), (1, None), (2, None)]),
    ((0, 2, 3), [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None), (2, None)]),
    ((1, 2, 1), [(0, None), (1, 0), (2, None)]),
    ((2, 3, 2), [(0, None), (1, None), (2, 0), (2, 1)]),
])
def test_the_order_of_layers_and_passes(loop, want):
    d = _dict()
    d.pop("loop")
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    cfg = RobuvikConfig.from_dict(d)
    assert list(cfg.run_order()) == want == plain.run_order(d)


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [
    (64, 1e4, 4.0, 300.0, 32.0, 1.0), (16, 500.0, 2.5, 60.0, 8.0, 2.0), (6, 150.0, 3.0, 40.0, 2.0, 2.0), (48, 2e4, 16.0, 2000.0, 64.0, 0.5),
    (8, 10.0, 5.0, 8.0, 40.0, 30.0), (10, 0.5, 2.0, 100.0, 3.0, 1.0)])
def test_stretched_rotary_frequencies(dims, base, factor, original, fast, slow):
    from vllm_oxide_b200.parts import YarnScaling, rotary_table
    got, mag = rotary_table(dims, base, YarnScaling(factor, original, fast, slow))
    want, wmag = plain.yarn(dims, base, dict(factor=factor, original=original, fast=fast, slow=slow))
    assert got.dtype.name == "float32" and len(got) == dims // 2 and abs(mag - wmag) < 1e-12
    assert torch.allclose(torch.from_numpy(got).double(), torch.tensor(want, dtype=torch.float64), rtol=1e-7, atol=0)
    flat, one = rotary_table(dims, base)
    assert one == 1.0 and abs(float(flat[1]) - base ** (-2 / dims)) < 1e-6 * base ** (-2 / dims)


def test_stretched_frequencies_by_hand():
    """Base e^8 over 8 features: ln(base) = 8, so the pair that turns n times over 2 pi e^3 positions has index (3 - ln n) / 2:
    1.5 for one turn (up to 2), 0.5 for e^2 turns (down to 0). Pair 0 keeps its frequency, pair 1 lies half way, 2 and 3 are divided."""
    from vllm_oxide_b200.parts import YarnScaling, rotary_table
    base, n = math.exp(8.0), 2 * math.pi * math.exp(3.0)
    got, mag = rotary_table(8, base, YarnScaling(4.0, n, math.exp(2.0), 1.0))
    f = [math.exp(-2.0 * i) for i in range(4)]
    want = [f[0], f[1] * (0.5 / 4 + 0.5), f[2] / 4, f[3] / 4]
    assert torch.allclose(torch.from_numpy(got).double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6)
    assert abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-12


# ------------------------------------------------------------------------------------ the plain model by hand
def test_plain_pair_rows():
    assert plain.bigram_rows([3, 5, 0], 23, 7, 5) == [23, (3 * 7 + 5 * 5) % 23, (5 * 7) % 23]


def test_plain_softmax_with_one_more():
    w = plain.softmax_off_by_one(torch.tensor([[0.0, math.log(2.0), -math.inf], [-200.0, -300.0, -400.0], [300.0, 300.0, 0.0]], dtype=torch.float64))
    assert torch.allclose(w[0], torch.tensor([0.25, 0.5, 0.0], dtype=torch.float64))
    assert float(w[1].sum()) < 1e-80 and torch.allclose(w[2], torch.tensor([0.5, 0.5, 0.0], dtype=torch.float64))


def test_plain_rotations_pair_features_as_they_should():
    x = torch.zeros(2, 1, 4, dtype=torch.float64)
    x[1, 0, 0] = 1.0
    rot = {"dims": 4, "base": 9.0}
    half, inter = plain.rotate(x, rot, False)[1, 0], plain.rotate(x, rot, True)[1, 0]
    assert torch.allclose(half, torch.tensor([math.cos(1), 0, math.sin(1), 0], dtype=torch.float64))
    assert torch.allclose(inter, torch.tensor([math.cos(1), math.sin(1), 0, 0], dtype=torch.float64))


def test_plain_window_counts_the_query_itself():
    assert plain.visible(4, 2).tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False],
                                            [False, False, True, True]]


def test_plain_experts_read_their_weight_times_the_input():
    t = {"router": torch.tensor([[0.0, 0.0], [10.0, 0.0]], dtype=torch.float64)}
    for e in range(2):
        for n in ("gate", "up", "down"):
            t[f"e{e}.{n}"] = torch.eye(2, dtype=torch.float64) * (e + 1)
    h = torch.tensor([[1.0, -2.0]], dtype=torch.float64)
    s = 1 / (1 + math.exp(-10.0))
    z = 2 * s * h
    want = 2 * (z * torch.sigmoid(z) * z)
    got = plain.moe_ff(h, t, "", {"router": {"experts": 2, "top": 1}})
    assert torch.allclose(got, want)
