"""Gogotar without a GPU: its configuration, plan, tensor list, cache needs and run order, the pages of a chunked layer, frequencies
slowed by wavelength, random-weights mode, and the plain implementation's pieces against each other."""
import json
import math

import numpy as np
import pytest
import torch

from kvad_b200 import write_random_model
from kvad_b200.cache import KVNeed
from kvad_b200.cache.pages import CacheError, SlotBook
from kvad_b200.config import ConfigError, JsonView, load_config, resolve
from kvad_b200.models.plan import LayerCall, Model
from kvad_b200.parts.base import PartSpec, build_part
from tests.gogotar_configs import CONFIGS, SEEDS
from tests.plain import gogotar_plain as pl


def typed(name):
    arch = resolve(JsonView(CONFIGS[name]))
    return arch, arch.read_config(JsonView(CONFIGS[name]))


def test_the_registry_finds_it_by_the_architecture_key():
    arch, c = typed("A")
    assert arch.id == "gogotar" and (c.width, c.embedding_scale, c.logit_softcap, c.loop) == (72, 2.5, 9.0, (1, 3, 2))
    assert typed("B")[1].logit_softcap is None and typed("C")[1].loop is None


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_plan_asks_for_exactly_the_tensors_the_writer_writes(tmp_path, name):
    d = write_random_model(str(tmp_path), CONFIGS[name], SEEDS[name])
    arch, cfg = load_config(d)
    stored = pl.read_tensors(str(tmp_path / "model.safetensors"))
    assert {r.name: tuple(r.shape) for r in Model(arch.plan(cfg)).requests()} == {k: tuple(v.shape) for k, v in stored.items()}
    written = json.load(open(tmp_path / "config.json"))
    assert {k: written[k] for k in CONFIGS[name]} == CONFIGS[name] and set(written) - set(CONFIGS[name]) <= {"torch_dtype"}
    assert pl.forward(*pl.load(d), [1, 2, 3]).shape == (3, CONFIGS[name]["vocab"])
    assert not [n for n in stored if n.endswith(("mix.v", "head"))]              # no value projection, no head of its own


def test_a_layer_without_a_feed_forward_has_no_second_norms():
    arch, c = typed("B")
    names = {r.name for r in Model(arch.plan(c)).requests()}
    assert {"l1.norm1", "l1.norm1b"} <= names and not {n for n in names if n.startswith(("l1.norm2", "l1.mlp"))}


def test_cache_needs_and_run_order_follow_the_loop():
    arch, c = typed("A")
    m = Model(arch.plan(c))
    lat0, att, lat2 = KVNeed(1, 24, None, value_dim=0), KVNeed(2, 16, None, value_dim=16, chunk=40), KVNeed(1, 40, None, value_dim=0)
    assert m.plan.order == tuple(LayerCall(layer, entry) for entry, layer in enumerate([0, 1, 2, 1, 2]))
    assert m.cache_layout.needs == (lat0, att, lat2, att, lat2)                  # every pass keeps what it wrote
    assert m.cache_layout.bytes_per_token(2) == 2 * (24 + 2 * (2 * 16 * 2 + 40))
    assert m.graph_safe and m.max_positions is None
    arch, c = typed("B")
    assert [call.layer for call in Model(arch.plan(c)).plan.order] == [0, 0, 0, 1, 2]
    arch, c = typed("S")
    assert [call.layer for call in Model(arch.plan(c)).plan.order] == [0, 1, 2, 1, 2, 1, 2] == pl.run_order(CONFIGS["S"])


def test_libraries_are_those_of_the_models_parts():
    from kvad_b200.ops import libraries_for
    arch, c = typed("A")
    libs = libraries_for(torch.bfloat16, Model(arch.plan(c)).kernel_families())
    assert {"norm_rotary", "attention_scored", "moe", "linear_tcgen05"} <= set(libs)
    assert not {"attention_prefill", "attention_decode", "attention_simt", "retention", "gated_recurrence", "channel_recurrence", "streams"} & set(libs)


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="convolution"), "type"),
    (lambda c: c.pop("embedding"), "scale"),
    (lambda c: c.pop("norm"), "eps"),
    (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "divide"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "size"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "pairs"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "pairs"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "experts"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "ff"),
    (lambda c: c["layers"][0].update(mlp={"kind": "routed", "ff": 8}), "mlp"),
    (lambda c: c["loop"].update(stop=4), "range"),
    (lambda c: c["loop"].update(times=0), "times"),
])
def test_a_configuration_that_cannot_be_run_is_refused(change, what):
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    change(cfg)
    arch = resolve(JsonView(cfg))
    with pytest.raises(ConfigError, match=what):
        arch.read_config(JsonView(cfg))


def test_frequencies_slowed_by_wavelength():
    """Pairs kept, pairs slowed by the whole factor and pairs between, against the plain function's."""
    for rot in ({"base": 3e4, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}},
                {"base": 50.0, "dims": 6, "scaling": {"factor": 2.0, "low": 0.8, "high": 5.0, "original": 40}},
                {"base": 1e5, "dims": 10, "scaling": {"factor": 3.0, "low": 2.0, "high": 2.0, "original": 100}}, {"base": 700.0, "dims": 12}):
        sc = rot.get("scaling")
        part = build_part("position", PartSpec("rotary", {"dims": rot["dims"], "base": rot["base"],
                                                          "scaling": {"kind": "wavelength", **sc} if sc else None}))

        class Fetch:
            device = "cpu"
        part.load_own(Fetch)
        want = pl.frequencies(rot)
        assert np.allclose(part.inv_freq.numpy(), want, rtol=1e-6) and part.mscale == 1.0
        if sc:
            plain = pl.frequencies({"base": rot["base"], "dims": rot["dims"]})
            assert np.isclose(want[0], plain[0]) and np.isclose(want[-1], plain[-1] / sc["factor"])
    between = (want := pl.frequencies({"base": 3e4, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}})) / \
        pl.frequencies({"base": 3e4, "dims": 64})
    assert ((between > 0.13) & (between < 0.99)).sum() >= 3 and (np.diff(want) < 0).all()
    with pytest.raises(ValueError, match="low"):
        build_part("position", PartSpec("rotary", {"dims": 4, "scaling": {"kind": "wavelength", "factor": 2.0, "high": 1.0, "original": 8}}))
    with pytest.raises(ValueError, match="kind"):
        build_part("position", PartSpec("rotary", {"dims": 4, "scaling": {"kind": "linear", "factor": 2.0, "original": 8}}))


@pytest.mark.parametrize("chunk", [1, 40, 64, 65, 200])
def test_a_chunked_group_keeps_what_the_next_positions_chunk_holds(chunk):
    """Every page that holds a position of the chunk of any row still to come is there; the others are back in the pool."""
    book = SlotBook(2, [16, 16], [None, None], page_size=64, chunks=[None, chunk])
    s = book.acquire()
    for step in [1, 1, 61, 1, 1, 62, 1, 1, 1, 70, 199, 1, 120]:
        book.grow(s, step)
        book.trim_windows(s)
        n = book.length[s]
        first = n // chunk * chunk
        for i, page in enumerate(book.pages[s][1]):
            assert (page >= 0) == ((i + 1) * 64 > first), (n, i)
        assert all(p >= 0 for p in book.pages[s][0])
        assert book.pools[1].n_out == sum(p >= 0 for p in book.pages[s][1])
    start = book.length[s] // chunk * chunk
    if start // 64 > 1:
        with pytest.raises(CacheError, match="dropped"):
            book.truncate(s, 64 - 1 if chunk > 64 else 63)
    assert book.truncate(s, max(start, book.length[s] - 1)) >= start
    book.release(s)
    book.check_all_free()
    with pytest.raises(ValueError, match="chunk"):
        KVNeed(1, 8, 5, chunk=7)


def test_a_layer_norm_takes_up_a_result_only_without_a_bias():
    spec = PartSpec("layernorm", {"width": 6, "eps": 1e-5, "bias": False, "name": ""})
    norm = build_part("norm", spec, "n")
    assert norm.takes_deferred and [r.name for r in norm.own_requests()] == ["n"]
    assert not build_part("norm", spec.with_params(bias=True), "n").takes_deferred
    mixer = PartSpec("latent_attention", {"width": 6, "n_heads": 1, "nope_dim": 4, "rot_dim": 0, "value_dim": 4, "q_rank": 4, "kv_rank": 4,
                                          "score_scale": 1.0, "norm_eps": 1e-5})
    assert build_part("block", PartSpec("sandwich", {"norm": spec, "mixer": mixer, "scaled": False}), "b.").centred
    with pytest.raises(ValueError, match="without a bias"):
        build_part("block", PartSpec("sandwich", {"norm": spec.with_params(bias=True), "mixer": mixer}), "b.")


def test_values_that_are_keys_leave_no_room_for_other_values():
    base = {"width": 16, "n_heads": 2, "key_dim": 8, "score_scale": 1.0, "v_name": None}
    part = build_part("mixer", PartSpec("shaped_score_attention", base), "m.")
    assert [r.name for r in part.requests()] == ["m.q", "m.k", "m.o"] and part.cache_need() == KVNeed(2, 8, None, value_dim=8)
    with pytest.raises(ValueError, match="keys"):
        build_part("mixer", PartSpec("shaped_score_attention", {**base, "value_dim": 4}), "m.")
    with pytest.raises(ValueError, match="chunk"):
        build_part("mixer", PartSpec("shaped_score_attention", {**base, "chunk": 4, "window": 4}), "m.")


def test_plain_mechanisms_agree_with_each_other():
    """The oracle's own pieces, checked against each other where the design says two things are the same."""
    rng = np.random.default_rng(0)
    T, H, d = 13, 2, 6
    q, k, v = (rng.standard_normal((T, H, d)) for _ in range(3))
    whole = pl.attend(q, k, v, 0.7, None, None, pl.chunk_mask(T, None))
    assert np.allclose(pl.attend(q, k, v, 0.7, None, np.full(H, -80.0), pl.chunk_mask(T, None)), whole)         # a sink that weighs nothing
    assert np.allclose(pl.attend(q, k, v, 0.7, None, np.full(H, 80.0), pl.chunk_mask(T, None)), 0.0)            # one that weighs everything
    assert np.allclose(pl.attend(q, k, v, 0.7, 1e6, None, pl.chunk_mask(T, None)), whole, atol=1e-6)            # a cap nothing comes near
    # a sink is one more key whose score is the sink and whose value is nothing
    sink = np.array([0.4, -1.2])
    got = pl.attend(q, k, v, 0.7, None, sink, pl.chunk_mask(T, None))
    for h in range(H):
        s = np.concatenate([q[-1, h] @ k[:, h].T * 0.7, [sink[h]]])
        e = np.exp(s)
        assert np.allclose(got[-1, h], (e[:-1] / e.sum()) @ v[:, h])
    # chunks: each is a sequence of its own; a chunk as long as the sequence is none; a chunk of one is the own value alone
    parts = np.concatenate([pl.attend(q[a:a + 5], k[a:a + 5], v[a:a + 5], 0.7, None, sink, pl.chunk_mask(len(q[a:a + 5]), None)) for a in (0, 5, 10)])
    assert np.allclose(pl.attend(q, k, v, 0.7, None, sink, pl.chunk_mask(T, 5)), parts)
    assert np.allclose(pl.attend(q, k, v, 0.7, None, None, pl.chunk_mask(T, T)), whole)
    assert np.allclose(pl.attend(q, k, v, 0.7, None, None, pl.chunk_mask(T, 1)), v)
    # scores of turned vectors depend on the distance only, and what does not turn passes
    rot = {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "low": 1.0, "high": 4.0, "original": 30}}
    a, b = rng.standard_normal((1, 1, d)), rng.standard_normal((1, 1, d))
    dots = [float((pl.turn(a, [p], rot) * pl.turn(b, [p - 3], rot)).sum()) for p in (3, 50)]
    assert math.isclose(dots[0], dots[1], rel_tol=1e-9) and np.array_equal(pl.turn(a, [9], rot)[..., 4:], a[..., 4:])
    # weights are the scores over all experts, not over the chosen ones
    z = rng.standard_normal((4, 7))
    c, w = pl.choose(z, 7)
    assert np.allclose(w.sum(-1), 1.0) and (pl.choose(z, 2)[1].sum(-1) < 1.0).all() and np.array_equal(pl.choose(z, 2)[0], c[:, :2])
    assert pl.choose(np.zeros((1, 5)), 2)[0].tolist() == [[0, 1]]
    # the clamped gate: level above the limit on the gate side, clamped on both sides for the other
    assert pl.clamped_glu(np.array([9.0]), np.array([0.3]), 2.0) == pl.clamped_glu(np.array([2.0]), np.array([0.3]), 2.0)
    assert pl.clamped_glu(np.array([1.0]), np.array([-7.0]), 2.0) == pl.clamped_glu(np.array([1.0]), np.array([-2.0]), 2.0)
    # layer norm: neither a shift nor a scale of the row shows
    x = rng.standard_normal((3, 9))
    assert np.allclose(pl.layer_norm(5.0 * x + 2.0, np.ones(9), 0.0), pl.layer_norm(x, np.ones(9), 0.0))
