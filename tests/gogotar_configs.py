"""Small Gogotar configurations for the tests: each differs from the others in every size, in the order of its layers and in which
options it has (a first layer of each kind; one key/value head for several heads, one each, or the key left out; a rotation over
part of a key or all of it, with frequencies slowed by wavelength - some pairs kept, some slowed, some between - or not; scores
capped or not; chunks of 1, 3, 40, a page, a page and one, several pages; no loop, a loop over one
layer, over all, from the first or up to the last; a router that takes one expert or all; a layer without a feed-forward; logits
capped or not; sizes that allow no 16-byte pieces)."""


def attention(heads, kv_heads, dim, chunk, rot_dims, base, scale=None, softcap=None, scaling=None, say_vdim=True):
    m = {"heads": heads, "dim": dim, "scale": scale or dim ** -0.5, "mask": {"size": chunk}, "rot": {"base": base, "dims": rot_dims}}
    if say_vdim:
        m["vdim"] = dim
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    if softcap is not None:
        m["softcap"] = softcap
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m}


def latent(heads, dim, vdim, q_rank, kv_rank, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "scale": scale or dim ** -0.5}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def model(width, vocab, scale, layers, mlps, eps=1e-5, cap=None, loop=None):
    out = {"architecture": "Gogotar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
           "layers": [{**layer, "mlp": mlp} for layer, mlp in zip(layers, mlps)]}
    if cap is not None:
        out["logit_softcap"] = cap
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # latent attention first; two layers run twice; three heads a key/value head; chunks shorter than a page
    "A": model(72, 257, 2.5,
               [latent(3, 12, 20, 28, 24), attention(6, 2, 16, 40, 8, 3e4, softcap=4.0, scaling=(3.0, 1.0, 5.0, 200)), latent(2, 24, 8, 16, 40, scale=0.4)],
               [dense(96, 0.9), moe(6, 2, 40), moe(8, 1, 16)], cap=9.0, loop=(1, 3, 2)),
    # attention first; no cap, no slowed frequencies, the whole key turns; the first layer runs three times; chunks of a page; uncapped logits
    "B": model(96, 500, 1.0,
               [attention(4, None, 24, 64, 24, 500.0), latent(5, 16, 16, 48, 32), attention(3, 1, 40, 3, 2, 1e3, scale=0.3, softcap=30.0)],
               [moe(9, 3, 32), None, dense(64, 3.0)], eps=1e-6, loop=(0, 1, 3)),
    # no loop; a page and one; a router that takes every expert; one head
    "C": model(128, 300, 0.7,
               [latent(8, 8, 48, 96, 64), attention(8, 4, 48, 65, 16, 1e5, softcap=12.0, scaling=(8.0, 2.0, 3.0, 64)), latent(1, 64, 32, 8, 88),
                attention(1, 1, 8, 200, 8, 20.0, scaling=(2.0, 0.5, 1.0, 4096), say_vdim=False)],
               [dense(128, 1.0), moe(4, 4, 64), moe(16, 2, 24), dense(40, 7.0)], cap=25.0),
    # sizes that are multiples of two at most: no product on the tensor cores, no 16-byte pieces anywhere
    "D": model(54, 131, 4.0,
               [attention(3, 3, 10, 33, 6, 900.0, softcap=3.0, scaling=(4.0, 1.0, 2.0, 32)), latent(3, 6, 10, 14, 18), attention(2, 1, 14, 7, 14, 50.0)],
               [moe(6, 2, 18), dense(30, 1.3), moe(5, 3, 14)], cap=5.0, loop=(0, 3, 2)),
    # every query sees its own key alone; a loop that ends with the last layer
    "S": model(80, 97, 1.5, [attention(4, 2, 12, 1, 4, 100.0, softcap=8.0), latent(4, 20, 4, 24, 48), attention(10, 2, 8, 127, 8, 1e4, softcap=50.0)],
               [dense(40, 2.0), moe(12, 5, 8), None], cap=30.0, loop=(1, 3, 3)),
    # larger and deeper: many small experts, chunks over several pages
    "E": model(320, 1000, 2.0,
               [attention(8, 4, 48, 300, 24, 1e4, softcap=15.0, scaling=(4.0, 1.0, 4.0, 512)), latent(6, 40, 56, 112, 96), attention(5, 5, 64, 130, 64, 5e5, softcap=20.0),
                latent(12, 24, 24, 64, 160)],
               [moe(32, 4, 64), dense(512, 1.5), moe(64, 6, 48), moe(12, 3, 96)], cap=30.0, loop=(1, 4, 2)),
}
SEEDS = {"A": 801, "B": 802, "C": 803, "D": 804, "S": 805, "E": 806}
#: the configurations every test of the engine runs on; "E" has tests of its own
SMALL = ("A", "B", "C", "D", "S")
