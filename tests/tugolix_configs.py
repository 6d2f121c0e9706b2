"""Small Tugolix configurations for the tests: each differs from the others in every size, in the order of its layers and in
which options it has (a first layer of each kind, one to five copies of the stream, one query/key head for several heads or the
key left out, one head, value columns that do not fill a block of the recurrence kernel, key sizes in several of its register
classes, a decay exponent of 1 and others, one to five taps, groups of one expert and one group of all, all groups kept or one,
a router that takes one expert or all, a layer without a feed-forward, a latent layer that reads another's cache, a logit scale
of 1 or left out, sizes that allow no 16-byte pieces)."""


def gla(heads, dim, vdim, tau, decay_rank=8):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": decay_rank}}


def latent(heads, dim, vdim, kv_rank, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale or dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def delta(heads, kv_heads, dim, vdim, conv, decay_rank=6, gate_rank=10):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank, "gate_rank": gate_rank}
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    return {"type": "channel_delta", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, count, keep, ff, limit, scale):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}},
            "expert": {"ff": ff, "limit": limit}}


def model(width, vocab, streams, layers, mlps, eps=1e-5, logit_scale=None):
    out = {"architecture": "Tugolix", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
           "layers": [{**layer, "mlp": mlp} for layer, mlp in zip(layers, mlps)]}
    if logit_scale is not None:
        out["logit_scale"] = logit_scale
    return out


CONFIGS = {
    # latent attention first; the last layer reads its cache; three copies; one group of all experts; all groups kept
    "A": model(64, 257, 3,
               [latent(3, 12, 20, 24), delta(4, 2, 16, 8, 3, 5, 7), gla(3, 8, 20, 4.0, 5), latent(2, 8, 6, 24, scale=0.5, kv_from=0)],
               [dense(96), moe(6, 2, 1, 1, 40, 1.5, 2.0), None, moe(8, 3, 4, 4, 16, 1.0, 0.7)], logit_scale=0.3),
    # gated linear attention first, one head, an exponent of 1; four copies; one query/key head for six heads; groups of one expert
    "B": model(96, 500, 4,
               [gla(1, 40, 48, 1.0, 16), delta(2, None, 24, 40, 2), latent(4, 16, 16, 32), delta(6, 1, 8, 16, 5, 9, 4), latent(2, 24, 8, 40),
                latent(5, 8, 24, 40, kv_from=4)],
               [moe(9, 1, 3, 1, 32, 2.0, 1.5), dense(64), None, moe(5, 2, 5, 3, 24, 0.5, 1.0), dense(200), moe(8, 4, 2, 1, 16, 1.0, 3.0)],
               eps=1e-6, logit_scale=1.0),
    # the delta rule first; key sizes in the recurrence kernel's larger register classes; two copies; no logit scale
    "C": model(128, 300, 2,
               [delta(2, 1, 136, 16, 4), gla(2, 72, 32, 9.0, 12), latent(8, 32, 32, 64), gla(4, 16, 8, 30.0)],
               [dense(128), moe(16, 2, 4, 2, 64, 1.0, 2.5), moe(2, 1, 1, 1, 96, 4.0, 1.2), dense(32)]),
    # sizes that are multiples of two at most: no product on the tensor cores, no 16-byte pieces anywhere; five copies
    "D": model(54, 131, 5,
               [delta(3, 3, 6, 10, 4, 3, 5), latent(3, 6, 10, 10), gla(2, 6, 18, 2.5, 3), latent(1, 10, 14, 10, kv_from=1)],
               [moe(6, 3, 3, 2, 18, 1.0, 1.8), dense(30), moe(4, 4, 2, 2, 14, 2.0, 0.5), None], logit_scale=2.0),
    # one copy; a latent layer reads the cache two layers back past one that keeps its own; one tap
    "S": model(72, 97, 1, [latent(4, 8, 12, 16), gla(5, 12, 6, 6.0, 7), latent(3, 20, 4, 48), latent(2, 10, 8, 16, kv_from=0), delta(2, 2, 12, 24, 1)],
               [None, dense(40), moe(12, 5, 3, 2, 8, 0.8, 1.1), dense(24), None], logit_scale=0.6),
    # larger and deeper: two latent layers with latents of their own, each read by a later layer; many small experts
    "E": model(320, 1000, 4,
               [latent(4, 48, 40, 96), gla(4, 48, 96, 12.0, 24), delta(4, 2, 96, 48, 3, 12, 20), latent(6, 32, 32, 96, kv_from=0),
                delta(8, 8, 32, 32, 4, 8, 8), latent(2, 64, 128, 160), gla(2, 128, 64, 20.0, 8), latent(8, 16, 16, 160, kv_from=5)],
               [moe(32, 4, 8, 3, 64, 1.0, 2.0), dense(512), moe(32, 4, 4, 2, 64, 1.0, 2.5), None, moe(12, 3, 6, 3, 96, 6.0, 1.0), dense(384),
                moe(64, 6, 8, 4, 48, 1.0, 2.5), moe(6, 2, 2, 1, 200, 2.0, 1.4)], logit_scale=0.5),
}
SEEDS = {"A": 701, "B": 702, "C": 703, "D": 704, "S": 705, "E": 706}
#: the configurations every test of the engine runs on; "E" has tests of its own
SMALL = ("A", "B", "C", "D", "S")
