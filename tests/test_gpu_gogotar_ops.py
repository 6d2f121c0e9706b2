"""The kernels behind Gogotar's mechanisms, each alone against the plain function of the same mechanism
(tests/plain/gogotar_plain.py, float64), at sizes of their own, with inputs made so that a fault shows: one key with e^40 times the
others' weight placed just inside and just outside a chunk (and behind the row), in a prompt and for a single row; sinks that weigh
nothing, everything and as much as the best key; rows far off centre whose layer norm a wrong mean would show; level router logits;
NaN-filled pages and buffers; shuffled pages."""
import numpy as np
import pytest
import torch

from kvad_b200.ops import KernelError, Ops
from tests.plain import gogotar_plain as pl
from tests.test_gpu_tugolix_ops import DT, dev, f32, i32, rel, stored

pytestmark = pytest.mark.gpu
KTOL = {"float32": 2e-5, "bfloat16": 8e-3}


def nan(shape, dtype):
    return torch.full(shape, float("nan"), device="cuda", dtype=dtype)


# ----------------------------------------------------------------------------- embedding and norms
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_rows_times_a_constant(dtype):
    rng, ops = np.random.default_rng(1), Ops(DT[dtype])
    table, toks = stored(rng.standard_normal((19, 36)), dtype), [4, 0, 18, 4, 7]
    out = nan((5, 36), torch.float32)
    ops.embed(i32(toks), i32(np.zeros(5)), dev(table, DT[dtype]), None, out, 2.75)
    assert rel(out, 2.75 * table[toks]) < 1e-7
    pos = stored(rng.standard_normal((9, 36)), dtype)                     # a position's row is not scaled
    ops.embed(i32(toks), i32([8, 0, 3, 3, 1]), dev(table, DT[dtype]), dev(pos, DT[dtype]), out, -0.5)
    assert rel(out, -0.5 * table[toks] + pos[[8, 0, 3, 3, 1]]) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [6, 54, 256, 512, 1000, 1024, 1030, 2048, 3072, 4096, 4100, 8192, 9001])
@pytest.mark.parametrize("centred_post,centred", [(True, True), (True, False), (False, True)])
def test_a_normed_result_enters_the_stream_and_the_next_sublayer_reads_it_normed(dtype, width, centred_post, centred):
    """Every register and shared-memory form; rows far off centre, a weight or none, all rows or listed ones, or the sum alone."""
    rng, ops, n, e1, e2 = np.random.default_rng(width), Ops(DT[dtype]), 9, 1e-3, 1e-5
    x, d = stored(rng.standard_normal((n, width)) * 2 + 5.0), stored(rng.standard_normal((n, width)) * np.exp(rng.uniform(-1.0, 3.0, (n, 1))) - 7.0)
    d[3] = 0.0                                                             # a row that nothing was added to
    g, w = stored(rng.standard_normal(width)), stored(1 + 0.3 * rng.standard_normal(width), dtype)

    def norm(c):
        return pl.layer_norm if c else pl.rms_norm
    new = x + norm(centred_post)(d, g, e1)
    want = norm(centred)(new, w, e2)
    xd, dd = f32(x), f32(d)
    rows, head = [7, 0, 7], nan((3, width), DT[dtype])
    args = dict(centred_post=centred_post, centred=centred)
    ops.sandwich_norm(xd, dd, f32(g), e1, head, dev(w, DT[dtype]), e2, rows=i32(rows), **args)          # a row list writes nothing back
    assert rel(head, want[rows]) < KTOL[dtype] and rel(xd, x) == 0.0 and rel(dd, d) == 0.0
    out = nan((n, width), DT[dtype])
    ops.sandwich_norm(xd, dd, f32(g), e1, out, dev(w, DT[dtype]), e2, **args)
    assert rel(out, want) < KTOL[dtype] and rel(xd, new) < 2e-6 and float(dd.abs().max()) == 0.0
    assert torch.equal(out[rows], head)                                    # a row's bits do not depend on its company
    dd.copy_(f32(d))
    ops.sandwich_norm(xd, dd, f32(g), e1, **args)                          # the sum alone
    assert rel(xd, new + norm(centred_post)(d, g, e1)) < 2e-6 and float(dd.abs().max()) == 0.0
    ops.sandwich_norm(xd, dd, f32(g), e1, out, None, e2, **args)           # nothing owed, no weight
    assert rel(out, norm(centred)(xd.double().cpu().numpy() + norm(centred_post)(np.zeros((n, width)), g, e1), 1.0, e2)) < KTOL[dtype]


def test_sandwich_norm_refuses_what_it_cannot_do():
    ops, x, g = Ops(torch.float32), torch.zeros((3, 8), device="cuda"), torch.ones(8, device="cuda")
    with pytest.raises(KernelError, match="row list"):
        ops.sandwich_norm(x, x.clone(), g, 1e-5, centred_post=True, centred=True, rows=i32([0]))
    with pytest.raises(KernelError, match="shape"):
        ops.sandwich_norm(x, torch.zeros((2, 8), device="cuda"), g, 1e-5, centred_post=True, centred=True)
    with pytest.raises(KernelError, match="as many"):
        ops.sandwich_norm(x, x.clone(), g, 1e-5, torch.empty((2, 8), device="cuda"), g, 1e-5, centred_post=True, centred=True)


# ----------------------------------------------------------------------------- attention
class Pages:
    """Keys and values of one sequence in shuffled pages among pages of NaNs."""

    def __init__(self, k, v, dtype, seed):
        n, G, dk = k.shape
        count = -(-n // 64)
        self.order = np.random.default_rng(seed).permutation(count + 3)[:count]
        self.table = i32(self.order)[None, :]
        self.kp, self.vp = (nan((count + 3, G, 64, a.shape[2]), DT[dtype]) for a in (k, v))
        for i in range(n):
            self.kp[int(self.order[i // 64]), :, i % 64] = dev(k[i], DT[dtype])
            self.vp[int(self.order[i // 64]), :, i % 64] = dev(v[i], DT[dtype])


def marked_queries(rng, k, H, chunk, weight):
    """Queries [n, H, dk] each of which one key answers far louder than all others: in turn the first and last key of the row's own
    chunk so far, the last of the chunk before it, a key behind the row, and its own."""
    n, G, dk = k.shape
    q = np.zeros((n, H, dk))
    for i in range(n):
        first = i // chunk * chunk
        for h in range(H):
            j = [first, max(first - 1, 0), i, min(i + 1, n - 1), max(first, i - 1), 0][(i + h) % 6]
            key = k[j, h // (H // G)]
            q[i, h] = key / (key @ key) * weight * (1.0 + 0.1 * rng.standard_normal())
    return q


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,chunk,cap", [(4, 4, 24, 24, 40, 0.0), (6, 2, 16, 20, 64, 9.0), (3, 1, 72, 72, 65, 60.0), (2, 2, 10, 6, 1, 5.0),
                                                 (8, 4, 32, 96, 3, 0.0), (5, 5, 14, 14, 127, 20.0), (2, 1, 128, 128, 200, 0.0)])
def test_chunks_sinks_caps_and_head_gates(dtype, H, G, dk, dv, chunk, cap):
    rng, ops, n, scale = np.random.default_rng(dk + chunk), Ops(DT[dtype]), 262, 0.5
    k, v = stored(rng.standard_normal((n, G, dk)), dtype), stored(rng.standard_normal((n, G, dv)), dtype)
    q = stored(marked_queries(rng, k, H, chunk, 40.0 / scale), dtype)
    sinks = stored(np.resize([-60.0, 3.0, 38.0, 0.0, 70.0], H))           # ... nothing, a little, as much as the marked key, everything
    gate = stored(rng.standard_normal((n, H)) * 2, dtype)
    want = pl.attend(q, k, v, scale, cap, sinks, pl.chunk_mask(n, chunk)) * pl.sigmoid(gate)[:, :, None]
    pages = Pages(k, v, dtype, dk)
    common = dict(softcap=cap, chunk=chunk, sinks=f32(sinks))
    got = nan((n, H * dv), DT[dtype])
    group = H // G
    ops.attention_scored(dev(q.reshape(n, -1), DT[dtype]), got, i32([0, n]), i32([n]), 1, n, pages.table, pages.kp, pages.vp, H, scale,
                         gate=dev(gate, DT[dtype]), heads_per_block=max(d for d in (1, 2, 4) if group % d == 0), **common)
    assert rel(got, want.reshape(n, -1)) < KTOL[dtype]
    # the tail of the prompt in a step of its own, beside nothing else
    tail = nan((7, H * dv), DT[dtype])
    ops.attention_scored(dev(q[n - 7:].reshape(7, -1), DT[dtype]), tail, i32([0, 7]), i32([n]), 1, 7, pages.table, pages.kp, pages.vp, H, scale,
                         gate=dev(gate[n - 7:], DT[dtype]), heads_per_block=1, **common)
    assert rel(tail, want[n - 7:].reshape(7, -1)) < KTOL[dtype]
    # single rows, keys whole or split over blocks (parts of which see no key at all)
    for i in sorted({0, 1, 63, 64, 65, chunk - 1, chunk, min(2 * chunk, n - 1), min(2 * chunk - 1, n - 1), 199, 261}):
        for splits in (1, 3, 6):
            one = nan((1, H * dv), DT[dtype])
            scratch = nan((H * splits * (dv + 2),), torch.float32) if splits > 1 else None
            ops.attention_scored(dev(q[i:i + 1].reshape(1, -1), DT[dtype]), one, i32([0, 1]), i32([i + 1]), 1, 1, pages.table, pages.kp, pages.vp, H, scale,
                                 gate=dev(gate[i:i + 1], DT[dtype]), heads_per_block=min(group, 32), n_splits=splits, scratch=scratch, **common)
            assert rel(one, want[i:i + 1].reshape(1, -1)) < KTOL[dtype], (i, splits)
    # the same without sinks and chunk: neither leaves a trace
    plain = nan((n, H * dv), DT[dtype])
    ops.attention_scored(dev(q.reshape(n, -1), DT[dtype]), plain, i32([0, n]), i32([n]), 1, n, pages.table, pages.kp, pages.vp, H, scale,
                         softcap=cap, heads_per_block=1)
    assert rel(plain, pl.attend(q, k, v, scale, cap, None, pl.chunk_mask(n, None)).reshape(n, -1)) < KTOL[dtype]


def test_a_key_outside_the_chunk_weighs_nothing_and_one_inside_all():
    """The marked key alone differs: moved across the edge, the output goes from its value to the sink's nothing."""
    ops, n, chunk = Ops(torch.float32), 200, 70
    k, v = np.zeros((n, 1, 4)), np.zeros((n, 1, 4))
    for j, mark in ((69, [1, 0]), (70, [0, 1])):
        k[j, 0, :2] = mark
        v[j, 0] = [*mark, 0.0, j]
    q = np.zeros((n, 2, 4))
    q[:, 0, 0] = q[:, 1, 1] = 60.0                                        # head 0 asks for key 69, head 1 for key 70
    pages = Pages(k, v, "float32", 3)
    out = nan((n, 8), torch.float32)
    ops.attention_scored(f32(q.reshape(n, -1)), out, i32([0, n]), i32([n]), 1, n, pages.table, pages.kp, pages.vp, 2, 1.0, chunk=chunk,
                         sinks=f32([0.0, 0.0]), heads_per_block=2)
    out = out.cpu().numpy().reshape(n, 2, 4)
    assert np.allclose(out[69, 0], v[69, 0]) and np.abs(out[70:, 0, 0]).max() == 0.0 and np.abs(out[:69, 0]).max() == 0.0
    assert np.allclose(out[70:140, 1], v[70, 0]) and np.abs(out[140:, 1]).max() == 0.0 and np.abs(out[:70, 1, 1]).max() == 0.0


def test_attention_refuses_sinks_and_chunks_it_cannot_take():
    ops, t = Ops(torch.float32), torch.zeros((1, 8), device="cuda")
    kp = torch.zeros((1, 1, 64, 8), device="cuda")
    args = (t, t.clone(), i32([0, 1]), i32([1]), 1, 1, i32([[0]]), kp, kp.clone(), 1, 1.0)
    with pytest.raises(KernelError, match="without a window"):
        ops.attention_scored(*args, chunk=4, window=4)
    with pytest.raises(KernelError, match="one per query head"):
        ops.attention_scored(*args, sinks=torch.zeros(2, device="cuda"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dim,rot", [(3, 3, 10, {"base": 40.0, "dims": 6, "scaling": {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 32}}),
                                         (8, 2, 48, {"base": 1e4, "dims": 48}), (4, 1, 16, {"base": 1e3, "dims": 4})])
def test_values_are_the_keys_before_their_norm_and_turn(dtype, H, G, dim, rot):
    """One buffer is key and value source of the store: the page of values gets the projection, the page of keys its norm, turned."""
    rng, ops, eps = np.random.default_rng(dim), Ops(DT[dtype]), 1e-4
    pos = np.array([0, 1, 62, 63, 64, 130])
    n = len(pos)
    buf = stored(rng.standard_normal((n, (H + G) * dim)) * 3, dtype)
    wq, wk = stored(1 + 0.3 * rng.standard_normal(dim)), stored(1 + 0.3 * rng.standard_normal(dim))
    q, k = buf[:, :H * dim].reshape(n, H, dim), buf[:, H * dim:].reshape(n, G, dim)
    bd = dev(buf, DT[dtype])
    order, kp, vp = [4, 0, 2], nan((6, G, 64, dim), DT[dtype]), nan((6, G, 64, dim), DT[dtype])
    keys = bd[:, H * dim:]
    ops.norm_turn_store(bd[:, :H * dim], keys, keys, i32(np.zeros(n)), i32(pos), i32([order]), kp, vp, H, q_weight=f32(wq), k_weight=f32(wk),
                        span_q=dim, span_k=dim, eps=eps, inv_freq=f32(pl.frequencies(rot)), dims=rot["dims"])
    want_q, want_k = pl.turn(pl.rms_norm(q, wq, eps), pos, rot), pl.turn(pl.rms_norm(k, wk, eps), pos, rot)
    assert rel(bd[:, :H * dim], want_q.reshape(n, -1)) < KTOL[dtype] and rel(bd[:, H * dim:], k.reshape(n, -1)) == 0.0
    for r, p in enumerate(pos):
        assert rel(kp[order[p // 64], :, p % 64], want_k[r]) < KTOL[dtype] and rel(vp[order[p // 64], :, p % 64], k[r]) == 0.0


# ----------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank,q_rank,n", [(40, 24, 70), (18, 14, 5), (96, 200, 33), (512, 8, 1)])
def test_both_latents_normed_in_one_launch(dtype, rank, q_rank, n):
    rng, ops, eps = np.random.default_rng(rank), Ops(DT[dtype]), 1e-4
    src, qs = (stored(rng.standard_normal((n, r + 6)) * 3, dtype) for r in (rank, q_rank))
    w, wq = stored(1 + 0.2 * rng.standard_normal(rank), dtype), stored(1 + 0.2 * rng.standard_normal(q_rank), dtype)
    kp, cq = nan((4, 1, 64, rank), DT[dtype]), nan((n, q_rank), DT[dtype])
    ops.latent_store(dev(src, DT[dtype])[:, :rank], dev(w, DT[dtype]), eps, None, i32(np.zeros(n)), i32(np.arange(n)), i32([[2, 0]]), kp, rank, 0,
                     interleaved=False, q_src=dev(qs, DT[dtype])[:, :q_rank], q_weight=dev(wq, DT[dtype]), q_out=cq)
    assert rel(kp[[2, 0]].reshape(-1, rank)[:n], pl.rms_norm(src[:, :rank], w, eps)) < KTOL[dtype]
    assert rel(cq, pl.rms_norm(qs[:, :q_rank], wq, eps)) < KTOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
# (heads up to 4, 8, 16 and more: single rows are dealt out to a block's warps accordingly; latents so long that a tile of 64 keys just fits, or does not)
@pytest.mark.parametrize("rank,H", [(40, 3), (64, 8), (22, 1), (264, 20), (512, 12), (100, 16), (505, 5)])
def test_shared_latents_with_a_sink_per_head(dtype, rank, H):
    """One far latent stands out; sinks from nothing to far above it; prompts and single rows."""
    rng, ops, n, scale = np.random.default_rng(rank), Ops(DT[dtype]), 200, 0.25
    c = stored(rng.standard_normal((n, 1, rank)), dtype)
    q = stored(marked_queries(rng, c, H, 64, 40.0 / scale), dtype)
    sinks = stored(np.resize([38.0, -60.0, 45.0, 1.0], H))
    want = pl.attend(q, c, c, scale, None, sinks, pl.chunk_mask(n, None)).reshape(n, -1)
    pages = Pages(c, c, dtype, rank)
    out = nan((n, H * rank), DT[dtype])
    ops.attention_scored(dev(q.reshape(n, -1), DT[dtype]), out, i32([0, n]), i32([n]), 1, n, pages.table, pages.kp, None, H, scale, value_dim=rank,
                         sinks=f32(sinks), heads_per_block=max(d for d in (1, 2, 4) if H % d == 0))
    assert rel(out, want) < KTOL[dtype]
    for i in (0, 63, 64, 199):
        for splits in (1, 4, 16):
            one = nan((1, H * rank), DT[dtype])
            scratch = nan((H * splits * (rank + 2),), torch.float32) if splits > 1 else None
            ops.attention_scored(dev(q[i:i + 1].reshape(1, -1), DT[dtype]), one, i32([0, 1]), i32([i + 1]), 1, 1, pages.table, pages.kp, None, H, scale,
                                 value_dim=rank, sinks=f32(sinks), heads_per_block=min(H, 32), n_splits=splits, scratch=scratch)
            assert rel(one, want[i:i + 1]) < KTOL[dtype], (i, splits)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,H,n_in,n_out", [(1, 3, 24, 20), (9, 5, 64, 40), (64, 2, 18, 10), (150, 4, 32, 48), (70, 3, 10, 14)])
def test_head_wise_maps_with_a_gate_per_entry(dtype, rows, H, n_in, n_out):
    rng, ops = np.random.default_rng(rows), Ops(DT[dtype])
    a, w = stored(rng.standard_normal((rows, H * n_in)), dtype), stored(rng.standard_normal((H, n_out, n_in)) / np.sqrt(n_in), dtype)
    gate = stored(rng.standard_normal((rows, H * n_out + 8)) * 2, dtype)
    want = np.einsum("hoi,rhi->rho", w, a.reshape(rows, H, n_in)).reshape(rows, -1) * pl.sigmoid(gate[:, 8:])
    out = nan((rows, H * n_out), DT[dtype])
    ops.linear_heads(dev(a, DT[dtype]), dev(w, DT[dtype]), out, head_stride_a=n_in, head_stride_out=n_out, gate=dev(gate, DT[dtype])[:, 8:])
    assert rel(out, want) < KTOL[dtype]


# ----------------------------------------------------------------------------- routing
def route(ops, z, top, scale=1.0):
    n, E = z.shape
    padded = f32(np.concatenate([z, np.full((n, 3), 1e9)], 1))[:, :E]        # (a view: what lies beside the logits is not one)
    chosen, weight = torch.full((n, top), -7, device="cuda", dtype=torch.int32), nan((n, top), torch.float32)
    tiles = ops.moe_max_tiles(n, top, E, 32)
    lists = [torch.empty(m, device="cuda", dtype=torch.int32) for m in (tiles, tiles * 32, tiles * 32, n * top)]
    ops.moe_sort(chosen, E, 32, *lists, logits=padded, weight=weight, routing="softmax", scale=scale)
    assert sorted(lists[3].cpu().tolist()) == sorted(np.nonzero(lists[2].cpu().numpy() >= 0)[0].tolist())       # every pair has its place
    return chosen.cpu().numpy(), weight


@pytest.mark.parametrize("E,top", [(6, 2), (8, 8), (16, 2), (17, 3), (130, 6), (512, 9), (1, 1), (5, 1), (64, 4)])
@pytest.mark.parametrize("n", [1, 33, 255, 300])
def test_softmax_scores_are_not_renormalised(E, top, n):
    """255 rows are routed inside the launch that groups them, 300 by one of their own; level and hugely different logits."""
    rng, ops = np.random.default_rng(E + n), Ops(torch.float32)
    z = stored(rng.standard_normal((n, E)) * 4)
    got, weight = route(ops, z, top)
    want, w = pl.choose(z, top)
    assert np.array_equal(got, want) and rel(weight, w) < 1e-5
    assert top == E or float(weight.sum(-1).max()) < 1.0
    got, weight = route(ops, np.zeros((n, E)), top, 2.5)                   # level: the lower index; times a constant
    assert np.array_equal(got, np.tile(np.arange(top), (n, 1))) and rel(weight, np.full((n, top), 2.5 / E)) < 1e-6
    z = np.zeros((n, E))
    z[:, E - 1], z[:, 0] = 90.0, -90.0
    got, weight = route(ops, z, top)
    assert (got[:, 0] == E - 1).all() and float((weight[:, 0] - 1.0).abs().max()) < 1e-6 if E > 1 else True


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,E,top,width,ff", [(1, 5, 2, 48, 24), (7, 3, 3, 54, 10), (90, 6, 1, 64, 40), (300, 8, 2, 64, 32), (13, 1, 1, 32, 16)])
def test_routed_experts_weighed_at_their_output(dtype, rows, E, top, width, ff):
    """Weight streams for few rows, tiles on the CUDA cores and (bfloat16, many pairs) on the tensor cores."""
    from kvad_b200.parts.base import PartSpec, build_part
    rng, ops = np.random.default_rng(rows), Ops(DT[dtype])
    w = {"m.router": stored(rng.standard_normal((E, width)) * 2 / np.sqrt(width), dtype)}
    for e in range(E):
        for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            w[f"m.e{e}.{name}"] = stored(rng.standard_normal(shape) * 1.5 / np.sqrt(shape[1]), dtype)
    part = build_part("feed_forward", PartSpec("gated_routed_mlp", {"width": width, "n_experts": E, "top": top, "hidden": ff}), "m.")
    part.load(lambda name, keep_f32=False, **kw: dev(w[name], DT[dtype]))
    routes = []

    class Ctx:
        def __init__(self):
            self.ops = ops

        def buffer(self, shape, dt=None):
            dt = dt or DT[dtype]
            return nan(shape, dt) if dt.is_floating_point else torch.full(shape, -12345, device="cuda", dtype=dt)
    inner = ops.moe_sort
    ops.moe_sort = lambda chosen, *a, **k: (inner(chosen, *a, **k), routes.append(chosen.cpu().numpy()))
    h, x = stored(rng.standard_normal((rows, width)), dtype), stored(rng.standard_normal((rows, width)))
    residual = f32(x)
    part.forward(Ctx(), dev(h, DT[dtype]), residual)
    want = x + pl.moe_ff(h, w, "m.", {"router": {"experts": E, "top": top}}, forced=routes[0])
    assert rel(residual, want) < (2e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_dense_feed_forward_clamps_both_sides(dtype):
    from kvad_b200.parts.base import PartSpec, build_part
    rng, ops, width, ff = np.random.default_rng(3), Ops(DT[dtype]), 40, 56
    w = {"m." + k: stored(rng.standard_normal(s) * 3 / np.sqrt(s[1]), dtype) for k, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    for limit in (0.4, 2.0, 50.0):
        part = build_part("feed_forward", PartSpec("clamped_glu_mlp", {"width": width, "hidden": ff, "limit": limit}), "m.")
        part.load(lambda name, keep_f32=False, **kw: dev(w[name], DT[dtype]))

        class Ctx:
            def __init__(self):
                self.ops = ops

            def buffer(self, shape, dt=None):
                return nan(shape, dt or DT[dtype])
        h, residual = stored(rng.standard_normal((11, width)), dtype), torch.zeros((11, width), device="cuda")
        part.forward(Ctx(), dev(h, DT[dtype]), residual)
        assert rel(residual, pl.dense_ff(h, w, "m.", limit)) < (1e-5 if dtype == "float32" else 1e-2), limit
