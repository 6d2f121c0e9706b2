"""Tugolix without a GPU: its configuration, plan, tensor list, cache needs and run order, sizes read from the checkpoint's
shapes, random-weights mode, and the plain implementation's pieces against each other."""
import json

import numpy as np
import pytest
import torch

from kvad_b200 import write_random_model
from kvad_b200.cache import KVNeed, StateNeed
from kvad_b200.config import ConfigError, JsonView, load_config, resolve
from kvad_b200.models.plan import LayerCall, Model
from kvad_b200.weights.safetensors_io import Checkpoint
from tests.plain import tugolix_plain as pl
from tests.tugolix_configs import CONFIGS, SEEDS

RANKS = ("decay_rank", "gate_rank")


def build(folder):
    """The model as `Engine.from_pretrained` builds it, short of the device."""
    arch, cfg = load_config(folder)
    ckpt = Checkpoint.open_dir(folder)
    try:
        cfg = arch.with_checkpoint_shapes(cfg, lambda n: tuple(ckpt.entries[n].shape) if n in ckpt.entries else None)
    finally:
        ckpt.close()
    return cfg, Model(arch.plan(cfg))


def test_the_registry_finds_it_by_the_architecture_key():
    arch = resolve(JsonView(CONFIGS["A"]))
    assert arch.id == "tugolix"
    c = arch.read_config(JsonView(CONFIGS["A"]))
    assert (c.width, c.streams, c.logit_scale) == (64, 3, 0.3)
    assert arch.read_config(JsonView(CONFIGS["C"])).logit_scale == 1.0       # (left out)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_plan_asks_for_exactly_the_tensors_the_writer_writes(tmp_path, name):
    d = write_random_model(str(tmp_path), CONFIGS[name], SEEDS[name])
    cfg, model = build(d)
    stored = pl.read_tensors(str(tmp_path / "model.safetensors"))
    assert {r.name: tuple(r.shape) for r in model.requests()} == {k: tuple(v.shape) for k, v in stored.items()}
    written = json.load(open(tmp_path / "config.json"))
    for got, typed, want in zip(written["layers"], cfg.layers, CONFIGS[name]["layers"]):
        assert not set(RANKS) & set(got["mixer"])                                        # the ranks are in the tensors' shapes only
        assert got["mixer"] == {k: v for k, v in want["mixer"].items() if k not in RANKS} and got["mlp"] == want["mlp"]
        assert typed["mixer"] == want["mixer"]                                           # ... and come back from there
    assert pl.forward(*pl.load(d), [1, 2, 3]).shape == (3, CONFIGS[name]["vocab"])


def test_a_layer_without_a_feed_forward_has_no_second_norm_or_connection():
    arch = resolve(JsonView(CONFIGS["A"]))
    names = {r.name for r in Model(arch.plan(arch.read_config(JsonView(CONFIGS["A"])))).requests()}
    assert {"l2.norm1", "l2.norm1.b", "l2.hc1.mix"} <= names and not {n for n in names if n.startswith(("l2.norm2", "l2.hc2", "l2.mlp"))}
    assert "l3.mix.dkv" not in names and "l3.mix.uk" in names                            # a latent layer that reads another's cache


def test_cache_needs_and_run_order_follow_the_layers(tmp_path):
    d = write_random_model(str(tmp_path), CONFIGS["A"], SEEDS["A"])
    _, model = build(d)
    needs = model.cache_layout.needs
    assert needs[0] == KVNeed(1, 24, None, value_dim=0)                    # the latent alone: no rotated part, no values
    assert needs[1] == StateNeed((4 * 8 * 16 + 2 * (2 * 2 * 16 + 4 * 8),), torch.float32)       # the matrices, and two kept inputs of q | k | v
    assert needs[2] == StateNeed((3 * 20 * 8,), torch.float32)
    assert len(needs) == 3                                                 # the last layer keeps nothing: it reads entry 0
    assert model.plan.order == (LayerCall(0, 0), LayerCall(1, 1), LayerCall(2, 2), LayerCall(3, 0, writes_cache=False))
    assert model.graph_safe and model.max_positions is None
    assert model.cache_layout.bytes_per_token(2) == 2 * 24


def test_libraries_are_those_of_the_models_parts():
    from kvad_b200.ops import libraries_for
    arch = resolve(JsonView(CONFIGS["A"]))
    libs = libraries_for(torch.bfloat16, Model(arch.plan(arch.read_config(JsonView(CONFIGS["A"])))).kernel_families())
    assert {"streams", "attention_scored", "gated_recurrence", "moe", "linear_tcgen05"} <= set(libs)
    assert not {"attention_prefill", "attention_decode", "attention_simt", "retention", "channel_recurrence"} & set(libs)


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="convolution"), "type"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.update(streams=40), "streams"),
    (lambda c: c["layers"][2]["mixer"].pop("tau"), "tau"),
    (lambda c: c["layers"][2]["mixer"].update(tau=0), "tau"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "divide"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "earlier"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "latent"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=16), "latent size"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "experts"),
    (lambda c: c["layers"][3]["mlp"]["router"].update(groups={"count": 3, "keep": 1}), "groups"),
    (lambda c: c["layers"][3]["mlp"]["router"].update(groups={"count": 4, "keep": 5}), "groups"),
    (lambda c: c["layers"][3]["mlp"]["router"].update(groups={"count": 4, "keep": 1}), "chosen from"),
    (lambda c: c["layers"][1]["mlp"]["router"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0].update(mlp={"kind": "routed", "ff": 8}), "mlp"),
    (lambda c: c.pop("norm"), "eps"),
])
def test_a_configuration_that_cannot_be_run_is_refused(change, what):
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    change(cfg)
    arch = resolve(JsonView(cfg))
    with pytest.raises(ConfigError, match=what):
        arch.read_config(JsonView(cfg))


def test_a_constant_in_front_of_the_logits_rides_in_the_final_norm():
    from kvad_b200.parts.base import PartSpec, build_part
    mats = {"n": torch.tensor([1.0, 2.0, 3.0]), "n.b": torch.tensor([0.5, 0.0, -1.0])}
    norm = build_part("norm", PartSpec("layernorm", {"width": 3, "eps": 1e-5, "name": "", "bias_name": ".b", "output_scale": 0.25}), "n")
    norm.load_own(lambda name, keep_f32=False: mats[name])
    gain, bias, centred, eps = norm.affine()
    assert gain.tolist() == [0.25, 0.5, 0.75] and bias.tolist() == [0.125, 0.0, -0.25] and centred and eps == 1e-5
    assert [r.name for r in norm.own_requests()] == ["n", "n.b"]


def test_plain_mechanisms_agree_with_each_other():
    """The oracle's own pieces, checked against each other where the design says two things are the same."""
    rng = np.random.default_rng(0)
    # copies mixed by the identity, each taking all of the result, are the plain residual sum
    x, y = rng.standard_normal((5, 4)), rng.standard_normal((5, 4))
    assert np.allclose(pl.write_streams(np.stack([x, x]), np.eye(2), np.ones(2), y), np.stack([x + y, x + y]))
    # the mix is indexed from, to
    assert np.allclose(pl.write_streams(np.stack([x, y]), np.array([[0.0, 1.0], [0.0, 0.0]]), np.zeros(2), y)[1], x)
    # the exponent: tau = 1 is the sigmoid, a large tau hardly forgets; the decay acts on the key's rows
    z = np.array([-2.0, 0.0, 3.0])
    assert np.allclose(pl.gla_decay(z, 1.0), pl.sigmoid(z)) and np.all(pl.gla_decay(z, 1e6) > 0.9999)
    T, dk, dv = 12, 5, 4
    q, k, v, a = rng.standard_normal((T, dk)), rng.standard_normal((T, dk)), rng.standard_normal((T, dv)), pl.sigmoid(rng.standard_normal((T, dk)))
    whole, _ = pl.gla_cell(q, k, v, a)
    first, S = pl.gla_cell(q[:5], k[:5], v[:5], a[:5])
    assert np.allclose(np.concatenate([first, pl.gla_cell(q[5:], k[5:], v[5:], a[5:], S)[0]]), whole)
    kept = np.cumprod(a[::-1], 0)[::-1]                      # by direct sum: what is left of key j at row t
    direct = sum((q[T - 1] * (kept[j + 1] if j + 1 < T else 1.0)) @ k[j] * v[j] for j in range(T))
    assert np.allclose(whole[-1], direct)
    # the delta rule with beta = 1, no decay and orthonormal keys stores and returns each value exactly
    keys, vals = np.eye(dk)[:4], rng.standard_normal((4, dv))
    out, S = pl.delta_cell(keys, keys, vals, np.ones(4), np.ones((4, dk)))
    assert np.allclose(out, vals) and np.allclose(S[:4], vals)
    # one group, or all groups kept: the largest choice scores; with no correction those are the largest logits
    z = rng.standard_normal((6, 8))
    for groups in ({"count": 1, "keep": 1}, {"count": 4, "keep": 4}):
        c, w = pl.choose(z, np.zeros(8), {"groups": groups, "top": 3, "scale": 2.0})
        assert np.array_equal(c, np.argsort(-z, -1)[:, :3]) and np.allclose(w.sum(-1), 2.0)
    # a group of two good experts beats one with the single best; the best expert is then out of reach; scores may be negative
    z = np.array([[9.0, -9.0, 2.0, 2.0]])
    r = {"groups": {"count": 2, "keep": 1}, "top": 1, "scale": 1.0}
    assert pl.choose(z, np.zeros(4), r)[0][0, 0] == 2
    assert pl.choose(z, np.array([-5.0, -5.0, -9.0, -9.0]), r)[0][0, 0] == 0
    # the weights are the scores without the correction
    c, w = pl.choose(np.zeros((1, 4)), np.array([0.3, 0.0, 0.1, 0.0]), {"groups": {"count": 1, "keep": 1}, "top": 2, "scale": 1.0})
    assert c.tolist() == [[0, 2]] and np.allclose(w, 0.5)
    # the clamped gate: level above the limit on the gate side, clamped on both sides for the other
    assert pl.clamped_glu(np.array([9.0]), np.array([0.3]), 2.0) == pl.clamped_glu(np.array([2.0]), np.array([0.3]), 2.0)
    assert pl.clamped_glu(np.array([1.0]), np.array([-7.0]), 2.0) == pl.clamped_glu(np.array([1.0]), np.array([-2.0]), 2.0)
