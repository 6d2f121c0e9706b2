"""The kernels behind Tugolix's mechanisms, each alone against the plain function of the same mechanism
(tests/plain/tugolix_plain.py, float64), at sizes of their own, over several sequences packed into one step with shuffled
slots, in portions down to one row, and with inputs made so that a fault shows: a first key in a channel that never decays and
that the last query asks for beside channels that forget at once, copies of very different sizes whose mixes swap them, groups
whose best expert must stay out of reach, scores that tie or are negative, one key among hundreds that stands out."""
import numpy as np
import pytest
import torch

from kvad_b200.ops import KernelError, Ops
from tests.plain import tugolix_plain as pl

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dev(a, dtype=None):
    t = torch.as_tensor(np.ascontiguousarray(a))
    return (t.to(dtype) if dtype is not None else t).to("cuda")


def f32(a):
    return dev(a, torch.float32)


def i32(a):
    return dev(np.asarray(a, dtype=np.int32))


def rel(got, ref):
    got, ref = np.asarray(got.detach().double().cpu()), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape and np.isfinite(got).all()
    return float(np.abs(got - ref).max() / max(np.abs(ref).max(), 1e-30))


def stored(a, dtype="float32"):
    """The values a tensor of the given dtype holds, as float64."""
    return torch.as_tensor(np.asarray(a)).to(DT[dtype]).double().numpy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dk,dv,tau", [(3, 20, 24, 1.0), (1, 72, 16, 7.0), (2, 8, 40, 3.0), (2, 200, 5, 24.0), (1, 320, 20, 11.0), (2, 30, 18, 2.0)])
def test_gated_linear_keeps_a_first_key_in_a_channel_that_does_not_decay(dtype, H, dk, dv, tau):
    rng, ops = np.random.default_rng(dk), Ops(DT[dtype])
    lens, slots, T = [300, 9, 1], [4, 0, 2], 300
    q, k, v = (stored(rng.standard_normal((3, T, H * d)), dtype) for d in (dk, dk, dv))
    z = stored(rng.standard_normal((3, T, H * dk)) * 3.0)
    z[0, :, 0::dk] = 80.0                     # channel 0 of every head never decays ...
    z[0, :, 1::dk] = -80.0 * tau              # ... channel 1 forgets at once
    k[0, 1:, 0::dk] = 0.0                     # only the first key has a part along channel 0,
    k[0, 0, 0::dk] = 1.0
    q[0, -1] = 0.0
    q[0, -1, 0::dk] = 3.0                     # and the last query asks for exactly it
    scale = 0.5
    want = [np.concatenate([pl.gla_cell(q[s, :n, a * dk:(a + 1) * dk] * scale, k[s, :n, a * dk:(a + 1) * dk], v[s, :n, a * dv:(a + 1) * dv],
                                        pl.gla_decay(z[s, :n, a * dk:(a + 1) * dk], tau))[0] for a in range(H)], axis=1) for s, n in enumerate(lens)]
    assert np.allclose(want[0][-1], 1.5 * v[0, 0])                    # what the first row wrote, 299 rows later
    for ready in (False, True):
        state = torch.zeros((6, ops.recurrence_state_size("gated_linear", H, dk, dv) + 3), device="cuda")
        done = [0, 0, 0]
        for portion in ([100, 9, 1], [1, 0, 0], [2, 0, 0], [197, 0, 0]):
            live = [s for s in range(3) if portion[s]]
            starts = np.concatenate([[0], np.cumsum([portion[s] for s in live])])
            cut = lambda a: np.concatenate([a[s, done[s]:done[s] + portion[s]] for s in live])
            out = torch.full((int(starts[-1]), H * dv), float("nan"), device="cuda")
            gates = f32(cut(z))
            if ready:                         # the decays in a pass of their own, as for prompts
                ops.power_gate(gates, tau)
                assert rel(gates, pl.gla_decay(cut(z), tau)) < 1e-6
            ops.gated_recurrence("gated_linear", dev(cut(q), DT[dtype]), dev(cut(k), DT[dtype]), dev(cut(v), DT[dtype]), gates, out, state, i32(starts),
                                 i32([slots[s] for s in live]), len(live), H, H, dk, dv, q_scale=scale, tau=tau, gates_ready=ready)
            for at, s in zip(starts, live):
                assert rel(out[at:at + portion[s]], want[s][done[s]:done[s] + portion[s]]) < 2e-5, (portion, s)
                done[s] += portion[s]
            if done[0] == 300:
                assert rel(out[-1:], want[0][-1:]) < 1e-6
        assert float(state[[1, 3, 5]].abs().max()) == 0.0          # slots of no sequence are untouched


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("act", ["silu", "sigmoid"])
def test_head_norm_with_a_shared_weight_and_either_gate(dtype, act):
    rng, ops, H, dv, eps = np.random.default_rng(5), Ops(DT[dtype]), 5, 18, 1e-3
    raw = stored(rng.standard_normal((9, H * dv)) * np.exp(rng.standard_normal((9, 1)) * 3))
    gate, w = stored(rng.standard_normal((9, H * dv)) * 2, dtype), stored(rng.standard_normal(dv), dtype)
    want = pl.rms_unit(raw.reshape(9, H, dv), eps) * w * {"silu": pl.silu, "sigmoid": pl.sigmoid}[act](gate).reshape(9, H, dv)
    out = torch.full((9, H * dv), float("nan"), device="cuda", dtype=DT[dtype])
    ops.head_norm_gate(f32(raw), dev(gate, DT[dtype]), dev(w, DT[dtype]), out, H, eps, weight_per_head=False, act=act)
    assert rel(out, want.reshape(9, -1)) < (1e-5 if dtype == "float32" else 6e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("copies,width", [(1, 64), (2, 54), (2, 1024), (3, 40), (3, 2052), (4, 1028), (4, 4100), (5, 96), (16, 30), (1, 8192), (4, 8200)])
@pytest.mark.parametrize("centred", [True, False])
def test_streams_read_mixed_and_normed_in_one_pass(dtype, copies, width, centred):
    """From the embedding output (all copies one tensor) through three sublayers to the head's rows: mixes that are no
    symmetric matrices and move copies about, shares and weights of both signs."""
    rng, ops, n, eps = np.random.default_rng(copies * width), Ops(DT[dtype]), 7, 1e-4
    x0 = stored(rng.standard_normal((n, width)) + 0.7)
    gain, bias = stored(1 + 0.3 * rng.standard_normal(width), dtype), stored(rng.standard_normal(width), dtype)
    tol = 2e-5 if dtype == "float32" else 6e-3

    def norm(u):
        return pl.layer_norm(u, gain, bias, eps) if centred else pl.rms_unit(u, eps) * gain + bias

    current, made = f32(x0), torch.full((copies, n, width), float("nan"), device="cuda")
    result = torch.zeros((n, width), device="cuda")
    ref, owed, ref_owed = np.stack([x0] * copies), None, None
    for layer in range(3):
        read, share, mix = (stored(rng.standard_normal(s)) for s in ((copies,), (copies,), (copies, copies)))
        out = torch.full((n, width), float("nan"), device="cuda", dtype=DT[dtype])
        ops.streams_norm(current, dev(gain, DT[dtype]), dev(bias, DT[dtype]), eps, out, centred=centred, copies=copies, read=f32(read), owed=owed,
                         x_out=made if owed else None)
        if owed is not None:
            ref = pl.write_streams(ref, *ref_owed)
            current = made
            assert rel(made, ref) < 1e-5 and float(result.abs().max()) == 0.0            # the new copies; what was owed is cleared
        u = pl.read_streams(ref, read)
        assert rel(out, norm(u)) < tol, layer
        y = stored(rng.standard_normal((n, width)) * 2)
        result += f32(y)
        owed, ref_owed = (result, f32(mix), f32(share)), (mix, share, y)
        # the last reader: the plain sum of what the copies will be, listed rows only, nothing written
        rows = [5, 0, 5, 3]
        head = torch.full((4, width), float("nan"), device="cuda", dtype=DT[dtype])
        before = current.clone()
        ops.streams_norm(current, dev(gain, DT[dtype]), dev(bias, DT[dtype]), eps, head, centred=centred, copies=copies, owed=owed, rows=i32(rows))
        assert rel(head, norm(pl.write_streams(ref, *ref_owed).sum(0))[rows]) < tol
        assert torch.equal(current, before) and rel(result, y) == 0.0
    if width % 4 == 0:                        # a row's bits do not depend on how many rows there are
        one = torch.empty((1, width), device="cuda", dtype=DT[dtype])
        ops.streams_norm(current, dev(gain, DT[dtype]), dev(bias, DT[dtype]), eps, one, centred=centred, copies=copies, owed=owed, rows=i32([3]))
        assert torch.equal(one[0], head[3])


def test_streams_refuse_what_they_cannot_do():
    ops, x, g = Ops(torch.float32), torch.zeros((3, 8), device="cuda"), torch.ones(8, device="cuda")
    out, owed = torch.empty((3, 8), device="cuda"), (torch.zeros((3, 8), device="cuda"), torch.eye(2, device="cuda"), torch.ones(2, device="cuda"))
    with pytest.raises(KernelError, match="place"):
        ops.streams_norm(x, g, None, 1e-5, out, centred=True, copies=2, owed=owed)
    with pytest.raises(KernelError, match="shape"):
        ops.streams_norm(x, g, None, 1e-5, out, centred=True, copies=3, owed=owed, x_out=torch.zeros((3, 3, 8), device="cuda"))
    with pytest.raises(KernelError, match="copies"):
        ops.streams_norm(x, g, None, 1e-5, out, centred=True, copies=17)


def route(ops, z, correction, router):
    n, E = z.shape
    top = router["top"]
    padded = f32(np.concatenate([z, np.full((n, 3), 1e9)], 1))[:, :E]        # (a view: what lies beside the logits is not one)
    chosen, weight = torch.full((n, top), -7, device="cuda", dtype=torch.int32), torch.full((n, top), float("nan"), device="cuda")
    tiles = ops.moe_max_tiles(n, top, E, 32)
    lists = [torch.empty(m, device="cuda", dtype=torch.int32) for m in (tiles, tiles * 32, tiles * 32, n * top)]
    ops.moe_sort(chosen, E, 32, *lists, logits=padded, weight=weight, routing="grouped_scores", correction=None if correction is None else f32(correction),
                 groups=(router["groups"]["count"], router["groups"]["keep"]), scale=router["scale"])
    assert sorted(lists[3].cpu().tolist()) == sorted(np.nonzero(lists[2].cpu().numpy() >= 0)[0].tolist())       # every pair has its place
    return chosen.cpu().numpy(), weight


@pytest.mark.parametrize("E,top,count,keep", [(6, 2, 1, 1), (8, 2, 4, 2), (8, 8, 2, 2), (5, 2, 5, 3), (130, 6, 10, 4), (512, 9, 256, 40), (36, 1, 3, 1), (16, 4, 4, 2), (1, 1, 1, 1)])
@pytest.mark.parametrize("n", [1, 33, 255, 300])
def test_grouped_choice_weights_and_ties(E, top, count, keep, n):
    """255 rows are routed inside the launch that groups them, 300 by one of their own."""
    rng, ops = np.random.default_rng(E + n), Ops(torch.float32)
    router = {"top": top, "groups": {"count": count, "keep": keep}, "scale": 1.7}
    z, correction = stored(rng.standard_normal((n, E)) * 2), stored(rng.standard_normal(E) * 0.3 - 0.6)      # (many choice scores are negative)
    c = pl.sigmoid(z) + correction
    clear = pl.routing_margin(z, correction, router) > 1e-5             # (64-bit and 32-bit scores may order level ones differently)
    got, weight = route(ops, z, correction, router)
    want, _ = pl.choose(z, correction, router)
    order = np.sort(np.take_along_axis(c, want, -1), -1)
    clear &= (np.diff(order, axis=-1).min(-1) if top > 1 else np.ones(n)) > 1e-6
    assert clear.sum() >= 0.9 * n
    assert np.array_equal(got[clear], want[clear])
    for row in got:
        assert len(set(row.tolist())) == top and row.min() >= 0 and row.max() < E
    assert rel(weight, pl.weigh(z, got, 1.7)) < 1e-6
    # level scores: the lower group, then the lower expert; no correction at all
    got, weight = route(ops, np.zeros((n, E)), None, router)
    assert np.array_equal(got, np.tile(np.arange(top), (n, 1))) and rel(weight, np.full((n, top), 1.7 / top)) < 1e-6


def test_the_best_expert_stays_out_of_reach_in_a_weak_group():
    ops = Ops(torch.float32)
    router = {"top": 2, "groups": {"count": 3, "keep": 1}, "scale": 1.0}
    z = np.array([[9.0, -9.0, -9.0, 1.0, 1.5, -9.0, 0.0, 0.5, 0.7]] * 2)
    got, w = route(ops, z, np.zeros(9), router)
    assert got.tolist() == [[4, 3]] * 2 and rel(w, pl.weigh(z, got, 1.0)) < 1e-6
    correction = np.array([0.0, 1.5, 0.0, 0.0, 0.0, 0.0, -2.0, -2.0, -2.0])       # the correction lifts the first group and steers the choice ...
    got, w = route(ops, z, correction, router)
    assert got.tolist() == [[1, 0]] * 2
    assert float(w[0, 0]) < 1e-3 and float(w[0, 1]) > 0.99                        # ... but not the weights


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank,H", [(40, 3), (64, 8), (22, 1)])
def test_latents_without_a_rotated_part_one_far_key_stands_out(dtype, rank, H):
    """The latent rows normed and stored alone; then a query that one key far back (the first, one at a page's border, the row's
    own) answers with e^30 times the weight of all others must read that key's latent and nothing else, for prompts and for single rows."""
    rng, ops, eps, n, scale = np.random.default_rng(rank), Ops(DT[dtype]), 1e-5, 260, 0.25
    pages = [7, 2, 5, 0, 3]
    src = stored(rng.standard_normal((n, rank + 6)) * 3, dtype)
    w = stored(1 + 0.2 * rng.standard_normal(rank), dtype)
    c = stored(pl.rms_unit(src[:, :rank], eps) * w, dtype)
    table, kp = i32(pages)[None, :], torch.full((8, 1, 64, rank), float("nan"), device="cuda", dtype=DT[dtype])
    ops.latent_store(dev(src, DT[dtype])[:, :rank], dev(w, DT[dtype]), eps, None, i32(np.zeros(n)), i32(np.arange(n)), table, kp, rank, 0, interleaved=False)
    flat = kp[pages].reshape(-1, rank)[:n]
    assert rel(flat, c) < (1e-6 if dtype == "float32" else 8e-3)
    c = flat.double().cpu().numpy()
    marks = [0, 63, 64, 127, 128, 191, 192, 255, 256, 259]
    q = np.zeros((n, H * rank))
    for i in range(n):
        for a in range(H):
            j = max(m for m in marks[:(i + a) % len(marks) + 1] if m <= i)
            others = np.abs(np.delete(c[:i + 1], j, 0) @ c[j]).max() if i else 0.0
            q[i, a * rank:(a + 1) * rank] = c[j] * (60.0 / scale / (c[j] @ c[j] - others if c[j] @ c[j] > others else c[j] @ c[j]))
    q = stored(q, dtype)
    want = np.zeros((n, H * rank))
    for a in range(H):
        s = np.where(np.tril(np.ones((n, n), dtype=bool)), q[:, a * rank:(a + 1) * rank] @ c.T * scale, -np.inf)
        want[:, a * rank:(a + 1) * rank] = pl.softmax_rows(s) @ c
    tol = 2e-5 if dtype == "float32" else 8e-3
    out = torch.full((n, H * rank), float("nan"), device="cuda", dtype=DT[dtype])
    ops.attention_scored(dev(q, DT[dtype]), out, i32([0, n]), i32([n]), 1, n, table, kp, None, H, scale, value_dim=rank,
                         heads_per_block=max(d for d in (1, 2, 4) if H % d == 0))
    assert rel(out, want) < tol
    for i in (0, 1, 63, 64, 65, 128, 200, 259):
        for splits in (1, 3):
            one = torch.full((1, H * rank), float("nan"), device="cuda", dtype=DT[dtype])
            scratch = torch.empty((H * splits * (rank + 2),), device="cuda") if splits > 1 else None
            ops.attention_scored(dev(q[i:i + 1], DT[dtype]), one, i32([0, 1]), i32([i + 1]), 1, 1, table, kp, None, H, scale, value_dim=rank,
                                 heads_per_block=min(H, 32), n_splits=splits, scratch=scratch)
            assert rel(one, want[i:i + 1]) < tol, (i, splits)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 5, 200])
def test_dense_feed_forward_with_a_bias_on_each_product(dtype, rows):
    from kvad_b200.parts.base import PartSpec, build_part
    rng, ops, width, ff = np.random.default_rng(rows), Ops(DT[dtype]), 48, 72
    w = {"m.gate": (ff, width), "m.up": (ff, width), "m.down": (width, ff), "m.gate.b": (ff,), "m.up.b": (ff,), "m.down.b": (width,)}
    w = {k: stored(rng.standard_normal(s) / (np.sqrt(s[-1]) if len(s) > 1 else 1.0), dtype) for k, s in w.items()}
    part = build_part("feed_forward", PartSpec("gated_mlp", {"width": width, "hidden": ff, "activation": "silu", "bias_suffix": ".b"}), "m.")
    part.load(lambda name, keep_f32=False, **kw: dev(w[name], DT[dtype]))

    class Ctx:
        def __init__(self):
            self.ops = ops

        def buffer(self, shape, dt=None):
            return torch.full(shape, float("nan"), device="cuda", dtype=dt or DT[dtype])
    h, x = stored(rng.standard_normal((rows, width)), dtype), stored(rng.standard_normal((rows, width)))
    residual = f32(x)
    part.forward(Ctx(), dev(h, DT[dtype]), residual)
    assert rel(residual, x + pl.dense_ff(h, w, "m.")) < (1e-5 if dtype == "float32" else 1e-2)
