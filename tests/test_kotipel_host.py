"""Host side of the Kotipel serving path on the CPU: configuration, registry, layer runs, cache layout, and that the
tests' models are sharp enough for a mistake in a mechanism to show."""

import copy
import math

import pytest
import torch

from flashrec_b200 import registry
from flashrec_b200.kotipel import KotipelConfig, random_tensors
from flashrec_b200.kvcache import PAGE, CacheSpec, LayerCaches, SequenceManager
from flashrec_b200.lm_layers import rotary_frequencies
from oracle import kotipel_oracle as O
from tests.kotipel_cases import CASES, make, tokens


def test_config_reads_sizes_and_loops():
    cfg = KotipelConfig.from_json(CASES["ragged"])
    assert [(r.layer, r.step) for r in cfg.runs()] == [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None), (2, None), (3, None)]
    shapes = cfg.tensor_shapes()
    assert shapes["l0.mix.in"] == (2 * 60 + 2 * 2 * 12 + 6, 90) and shapes["l0.mix.conv"] == (60 + 48, 3)
    assert shapes["l1.mix.left.k"] == (2 * 20, 90) and shapes["l1.mix.right.a1"] == (None, 90)
    assert "l2.mlp.gate" not in shapes and "l2.norm2" not in shapes and shapes["side.embed"] == (131, 4 * 11)
    specs = cfg.cache_specs()
    assert len(specs) == 8 and specs[0] == specs[2] and (specs[0].k_cols, specs[0].mask) == (0, "none")
    assert (specs[1].k_cols, specs[1].v_cols, specs[1].state_floats) == (2 * 32, 2 * 32, 3 * 24 * 32)
    for name, raw in CASES.items():
        assert [(r.layer, r.step) for r in KotipelConfig.from_json(raw).runs()] == O.run_order(raw), name
    assert "side.embed" not in KotipelConfig.from_json(CASES["single_kv"]).tensor_shapes()


def test_config_rejects_what_the_design_does_not_have():
    for change in (lambda c: c["layers"][0].update(type="mamba3"), lambda c: c["layers"][0]["mlp"].update(kind="mixture"),
                   lambda c: c.update(loop=dict(start=1, stop=9, times=2))):
        bad = copy.deepcopy(CASES["equal"])
        change(bad)
        with pytest.raises(ValueError):
            KotipelConfig.from_json(bad)


def test_registry_picks_the_family():
    assert registry.lookup(CASES["equal"]).name == "kotipel"
    assert torch.float32 in registry.lookup(CASES["equal"]).dtypes


def test_rotary_frequencies_blend_between_the_two_wavelengths():
    for rot in (dict(dims=24, base=5000.0, scaling=dict(factor=8.0, low=1.0, high=4.0, original=64)), dict(dims=10, base=1e6),
                dict(dims=64, base=30.0, scaling=dict(factor=3.0, low=0.5, high=7.0, original=40))):
        got = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling")).double().sum(1)
        assert torch.allclose(got, torch.tensor(O.rotary_frequencies(rot), dtype=torch.float64), rtol=1e-13)
    plain = rotary_frequencies(24, 5000.0).double().sum(1)
    scaled = rotary_frequencies(24, 5000.0, dict(factor=8.0, low=1.0, high=4.0, original=64)).double().sum(1)
    lengths = 2 * math.pi / plain
    assert torch.equal(scaled[lengths < 16], plain[lengths < 16]) and (lengths < 16).any()
    assert torch.allclose(scaled[lengths > 64] * 8, plain[lengths > 64]) and (lengths > 64).any()
    between = (lengths > 16) & (lengths < 64)
    assert between.any() and (scaled[between] < plain[between]).all() and (scaled[between] > plain[between] / 8).all()


def test_state_memory_and_pages(lib):
    cfg = KotipelConfig.from_json(CASES["ragged"])
    caches = LayerCaches(cfg.cache_specs(), 3, 4, torch.bfloat16, "cpu")
    assert caches.state[0].shape == (4, 6 * 16 * 16) and caches.state[0].dtype == torch.float32
    assert caches.k[0].shape == (3 * PAGE, 0) and caches.k[1].shape == (3 * PAGE, 64)
    for dim, vdim in ((12, 10), (8, 16), (33, 100)):
        assert CacheSpec(0, 0, state_heads=3, state_dim=dim, state_vdim=vdim).state_floats == 3 * lib.fr_linear_state_floats(dim, vdim)
    # a full-attention layer keeps every page, recurrent layers alone keep none but the current one
    full = SequenceManager(cfg.cache_specs(), 9, 1, 4000, "cpu")
    full.open(0)
    full.extend(0, 300)
    assert full.trim(0) == 0
    rec = SequenceManager(KotipelConfig.from_json(CASES["recurrent"]).cache_specs(), 3, 1, 4000, "cpu")
    rec.open(0)
    for _ in range(40):
        rec.extend(0, 50)
        rec.trim(0)
        assert len(rec.live[0].pages) <= 1
    assert CASES["recurrent"]["layers"][0]["type"] == "mamba2" and rec.specs[0].max_keys(100) == 0


def _fault(raw, w, what):
    bad, w = copy.deepcopy(raw), dict(w)
    left = [e["mixer"]["left"] for e in bad["layers"] if e["type"] == "parallel"]
    right = [e["mixer"]["right"] for e in bad["layers"] if e["type"] == "parallel"]
    if what == "rotation":
        left[0]["rot"]["dims"] -= 2
    if what == "scaling":
        left[0]["rot"]["scaling"]["factor"] += 1
    if what == "score":
        left[0]["scale"] *= 1.2
    if what == "tau":
        right[0]["tau"] *= 1.5
    if what == "limit":
        bad["layers"][0]["mlp"]["limit"] *= 1.3
    if what == "norm_groups":
        bad["layers"][0]["mixer"]["norm_groups"] //= 2
    if what == "pass":
        w["loop.step"] = w["loop.step"].flip(0)
    if what == "token":
        w["side.embed"] = w["side.embed"].roll(1, 0)
    for name in ("l0.mix.D", "l0.mix.conv.b", "l1.mix.left.g", "l1.mix.right.out", "l0.side.norm"):
        if what == name:
            w[name] = torch.zeros_like(w[name])
    return bad, w


@pytest.mark.parametrize("what", ["rotation", "scaling", "score", "tau", "limit", "norm_groups", "pass", "token", "l0.mix.D",
                                  "l0.mix.conv.b", "l1.mix.left.g", "l1.mix.right.out", "l0.side.norm"])
def test_a_planted_mistake_shows_in_the_oracle(what):
    raw, cfg, w = make("ragged")
    t = tokens(cfg, 70)
    good, bad = O.forward(raw, w, t), O.forward(*_fault(raw, w, what), t)
    err = ((good - bad)[30:].pow(2).mean(1) / good[30:].pow(2).mean(1)).sqrt()
    assert err.max() > 0.02, err.max()


@pytest.mark.parametrize("name", list(CASES))
def test_oracle_is_causal_and_remembers(name):
    raw, cfg, w = make(name)
    t = tokens(cfg, 40)
    full = O.forward(raw, w, t)
    assert torch.allclose(full[:15], O.forward(raw, w, t[:15]), atol=1e-4)
    other = list(t)
    other[3] = (t[3] + 1) % cfg.vocab  # a token far back still shows: the state or the cache holds it
    assert ((O.forward(raw, w, other) - full)[30:].abs().max(1).values > 1e-4).all()


def test_random_tensors_have_the_checkpoint_shapes():
    cfg = KotipelConfig.from_json(CASES["equal"])
    w = random_tensors(cfg, rank=7)
    assert set(w) == set(cfg.tensor_shapes()) and w["l1.mix.right.a1"].shape == (7, 128) and w["l1.mix.right.a2"].shape == (128, 7)
