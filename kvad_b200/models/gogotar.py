"""Gogotar: a decoder of `sandwich` blocks with layer norms, a range of which may run several times in a row.

    x = scale * embed[token]
    per layer:  x = x + norm1b(mixer(norm1(x)));  x = x + norm2b(mlp(norm2(x)))          (mlp may be absent)
    layers `loop.start` .. `loop.stop` - 1 run `loop.times` times with the same weights, every pass with cache entries of its own
    logits = cap * tanh(embed . norm(x) / cap)                                           (the table without its scale)

Norms are layer norms with a weight and no bias.  The mixer of a layer is `attention` (grouped heads; the values are the keys as
projected, before their norm and turn; queries and keys RMS-normed head by head; rotary pairs half apart whose frequencies may be
slowed by wavelength; capped scores; every query confined to its own chunk of positions; one sigmoid gate per head) or
`latent_attention` (queries through one low-rank latent, keys and values through another, which alone is cached; no positions;
an entry-wise sigmoid gate).  Both have a sink per head in the softmax's denominator.  The feed-forward is `dense` (the clamped
gated form) or `moe`: silu-gated experts, the `top` largest softmax scores chosen and weighing in as they are.

config.json: `architecture`, `vocab`, `width`, `embedding.scale`, `norm.eps`, `logit_softcap` (absent: none), `loop`: {`start`,
`stop`, `times`} or absent, and `layers`, a list of {`type`, `mixer`, `mlp`}.  `attention`: `heads`, `kv_heads` (absent: as many),
`dim`, `vdim` (as long as `dim`), `scale`, `softcap` (absent: none), `mask.size`, `rot`: {`base`, `dims`, `scaling`: {`factor`,
`low`, `high`, `original`} or absent}.  `latent_attention`: `heads`, `dim`, `vdim`, `q_rank`, `kv_rank`, `scale`.  `mlp`: null,
{`kind`: "dense", `ff`, `limit`} or {`kind`: "moe", `router`: {`experts`, `top`}, `expert`: {`ff`}}.  Tensors: `embed`,
`l<i>.norm1|norm1b|norm2|norm2b`, `l<i>.mix.<name>`, `l<i>.mlp.<name>`, `final.norm`; matrices are `[out, in]`.  This module only
describes: the configuration, the plan (which parts, with which sizes and tensor names, in which order with which cache entries)
and the random-weights recipe; all computing is in the parts.
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass
from typing import Optional

from ..config.json_view import ConfigError, JsonView
from ..config.registry import Architecture, register
from ..parts.base import PartSpec
from .plan import LayerCall, ModelPlan

MIXER_TYPES = ("attention", "latent_attention")


@dataclass(frozen=True)
class GogotarConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    logit_softcap: Optional[float]
    layers: tuple            # of dicts {"type", "mixer", "mlp"} as config.json has them
    loop: Optional[tuple]    # (start, stop, times) or None
    arch_id: str = "gogotar"


def _need(d, key: str, where: str, kinds=(int, float)):
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, kinds):
        raise ConfigError(f"config: {where} has no `{key}`")
    return v


def _pos_int(d, key: str, where: str) -> int:
    v = _need(d, key, where, (int,))
    if v <= 0:
        raise ConfigError(f"config: {where}: `{key}` must be positive")
    return int(v)


def _positive(d, key: str, where: str) -> float:
    v = _need(d, key, where)
    if not v > 0:
        raise ConfigError(f"config: {where}: `{key}` must be positive")
    return float(v)


def _check_attention(m: dict, where: str) -> None:
    heads = _pos_int(m, "heads", where)
    kv = _pos_int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    if heads % kv:
        raise ConfigError(f"config: {where}: {heads} heads do not divide into {kv} key/value heads")
    dim = _pos_int(m, "dim", where)
    if m.get("vdim") is not None and _pos_int(m, "vdim", where) != dim:
        raise ConfigError(f"config: {where}: the values are the keys, so `vdim` is `dim`")
    _need(m, "scale", where)
    if m.get("softcap") is not None:
        _positive(m, "softcap", where)
    _pos_int(m.get("mask"), "size", where + " mask")
    rot = m.get("rot")
    _positive(rot, "base", where + " rot")
    dims = _pos_int(rot, "dims", where + " rot")
    if dims % 2 or dims > dim:
        raise ConfigError(f"config: {where}: the rotation turns pairs: an even number of entries, at most a key's")
    if rot.get("scaling") is not None:
        for key in ("factor", "low", "high", "original"):
            _positive(rot["scaling"], key, where + " rot.scaling")


def read_config(view: JsonView) -> GogotarConfig:
    tree = view.tree
    vocab, width = _pos_int(tree, "vocab", "the model"), _pos_int(tree, "width", "the model")
    scale = float(_need(tree.get("embedding"), "scale", "`embedding`"))
    eps = float(_need(tree.get("norm"), "eps", "`norm`"))
    cap = _positive(tree, "logit_softcap", "the model") if tree.get("logit_softcap") is not None else None
    layers = tree.get("layers")
    if not isinstance(layers, list) or not layers:
        raise ConfigError("config: `layers` must be a non-empty list")
    for i, layer in enumerate(layers):
        where = f"layer {i}"
        if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
            raise ConfigError(f"config: {where}: `type` must be one of {MIXER_TYPES}")
        m = layer.get("mixer")
        if not isinstance(m, dict):
            raise ConfigError(f"config: {where} has no `mixer`")
        if layer["type"] == "attention":
            _check_attention(m, where)
        else:
            for key in ("heads", "dim", "vdim", "q_rank", "kv_rank"):
                _pos_int(m, key, where)
            _need(m, "scale", where)
        mlp = layer.get("mlp")
        if mlp is not None:
            if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
                raise ConfigError(f"config: {where}: `mlp` is null or of kind `dense` or `moe`")
            if mlp["kind"] == "dense":
                _pos_int(mlp, "ff", where + " mlp")
                _positive(mlp, "limit", where + " mlp")
            else:
                r = mlp.get("router")
                if _pos_int(r, "top", where + " router") > _pos_int(r, "experts", where + " router"):
                    raise ConfigError(f"config: {where}: more experts a token than experts")
                _pos_int(mlp.get("expert"), "ff", where + " expert")
    loop, span = tree.get("loop"), None
    if loop is not None:
        start, stop = _need(loop, "start", "`loop`", (int,)), _need(loop, "stop", "`loop`", (int,))
        times = _pos_int(loop, "times", "`loop`")
        if not (0 <= start < stop <= len(layers)):
            raise ConfigError("config: `loop` must name a range of layers")
        span = (int(start), int(stop), times)
    return GogotarConfig(vocab=vocab, width=width, embedding_scale=scale, norm_eps=eps, logit_softcap=cap,
                         layers=tuple(copy.deepcopy(layers)), loop=span)


def write_config(c: GogotarConfig) -> dict:
    out = {"architecture": "Gogotar", "vocab": c.vocab, "width": c.width, "embedding": {"scale": c.embedding_scale},
           "norm": {"eps": c.norm_eps}, "layers": copy.deepcopy(list(c.layers))}
    if c.logit_softcap is not None:
        out["logit_softcap"] = c.logit_softcap
    if c.loop:
        out["loop"] = {"start": c.loop[0], "stop": c.loop[1], "times": c.loop[2]}
    return out


def _mixer_spec(c: GogotarConfig, layer: dict) -> PartSpec:
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return PartSpec("latent_attention", {
            "width": c.width, "n_heads": m["heads"], "nope_dim": m["dim"], "rot_dim": 0, "value_dim": m["vdim"], "q_rank": m["q_rank"],
            "kv_rank": m["kv_rank"], "score_scale": m["scale"], "norm_eps": c.norm_eps, "sink_name": "sink", "gate_name": "g"})
    rot, scaling = m["rot"], m["rot"].get("scaling")
    return PartSpec("shaped_score_attention", {
        "width": c.width, "n_heads": m["heads"], "n_kv_heads": m.get("kv_heads") or m["heads"], "key_dim": m["dim"], "v_name": None,
        "score_scale": m["scale"], "softcap": m.get("softcap"), "chunk": m["mask"]["size"], "sink_name": "sink", "gate": "head",
        "position": PartSpec("rotary", {"dims": rot["dims"], "base": rot["base"], "layout": "half",
                                        "scaling": {"kind": "wavelength", **scaling} if scaling else None}),
        "qk_norm": {"span": "head", "eps": c.norm_eps}, "decode_blocks_per_sm": 4})


def _mlp_spec(c: GogotarConfig, mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("clamped_glu_mlp", {"width": c.width, "hidden": mlp["ff"], "limit": mlp["limit"], "alpha": 1.702})
    r = mlp["router"]
    return PartSpec("gated_routed_mlp", {"width": c.width, "n_experts": r["experts"], "top": r["top"], "hidden": mlp["expert"]["ff"],
                                         "activation": "silu", "routing": "softmax", "scores_at": "output"})


def run_order(c: GogotarConfig) -> list:
    """The layers in the order they run."""
    n = len(c.layers)
    if not c.loop:
        return list(range(n))
    start, stop, times = c.loop
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


def plan(c: GogotarConfig) -> ModelPlan:
    norm = PartSpec("layernorm", {"width": c.width, "eps": c.norm_eps, "bias": False, "name": ""})
    blocks = tuple(PartSpec("sandwich", {"norm": norm, "mixer": _mixer_spec(c, layer), "feed_forward": _mlp_spec(c, layer.get("mlp")),
                                         "scaled": False}) for layer in c.layers)
    kinds = "".join({"attention": "a", "latent_attention": "l"}[layer["type"]] for layer in c.layers)
    looped = f" · layers {c.loop[0]}..{c.loop[1] - 1} x {c.loop[2]}" if c.loop else ""
    return ModelPlan(
        arch_id="gogotar", vocab_size=c.vocab, width=c.width,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "width": c.width, "name": "embed", "scale": c.embedding_scale}),
        blocks=blocks, block_prefixes=tuple(f"l{i}." for i in range(len(blocks))),
        head=PartSpec("lm_head", {"vocab_size": c.vocab, "width": c.width, "norm": norm, "tied": True, "norm_name": "final.norm",
                                  "softcap": c.logit_softcap}),
        order=tuple(LayerCall(layer, entry) for entry, layer in enumerate(run_order(c))),      # every run has a cache entry of its own
        max_positions=None,
        summary=f"gogotar · {len(blocks)} layers ({kinds}){looped} · {c.width} wide · {c.vocab} vocab",
    )


def random_tensors(c: GogotarConfig, rng) -> dict:
    """Matrices ~N(0, 1/in), the embedding ~N(0, 1), norm weights near 1, sinks around 0 with a spread of 1."""
    def mat(out, inp, gain=1.0):
        return rng.normal((out, inp), gain / math.sqrt(inp))

    def near_one(n):
        return rng.normal((n,), 0.1, 1.0)

    w = c.width
    t = {"embed": rng.normal((c.vocab, w), 1.0), "final.norm": near_one(w)}
    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer["mixer"]
        t[p + "norm1"], t[p + "norm1b"] = near_one(w), near_one(w)
        H = m["heads"]
        t[p + "mix.sink"] = rng.normal((H,), 1.0)
        if layer["type"] == "attention":
            G, dk = m.get("kv_heads") or H, m["dim"]
            t[p + "mix.q"], t[p + "mix.k"] = mat(H * dk, w), mat(G * dk, w)
            t[p + "mix.q.norm"], t[p + "mix.k.norm"] = near_one(dk), near_one(dk)
            t[p + "mix.g"], t[p + "mix.o"] = mat(H, w, 2.0), mat(w, H * dk)
        else:
            dk, dv, rq, rk = m["dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            t[p + "mix.dq"], t[p + "mix.dq.norm"], t[p + "mix.uq"] = mat(rq, w), near_one(rq), mat(H * dk, rq, 1.5)
            t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = mat(rk, w), near_one(rk)
            t[p + "mix.uk"], t[p + "mix.uv"] = mat(H * dk, rk, 1.5), mat(H * dv, rk)
            t[p + "mix.g"], t[p + "mix.o"] = mat(H * dv, w, 2.0), mat(w, H * dv)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        t[p + "norm2"], t[p + "norm2b"] = near_one(w), near_one(w)
        if mlp["kind"] == "dense":
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(mlp["ff"], w, 1.5), mat(mlp["ff"], w, 1.5), mat(w, mlp["ff"])
            continue
        ff = mlp["expert"]["ff"]
        for e in range(mlp["router"]["experts"]):
            t[p + f"mlp.e{e}.gate"], t[p + f"mlp.e{e}.up"], t[p + f"mlp.e{e}.down"] = mat(ff, w, 1.5), mat(ff, w, 1.5), mat(w, ff)
        t[p + "mlp.router"] = mat(mlp["router"]["experts"], w, 2.0)
    return t


ARCH = register(Architecture(
    id="gogotar", model_types=("gogotar",),
    about="Gogotar: sandwich blocks with layer norms; chunked attention whose values are its keys, or latent attention, both with sinks and gates; "
          "dense or softmax-routed feed-forward; a repeated range of layers; capped logits from the embedding table",
    read_config=read_config, plan=plan, write_config=write_config, random_tensors=random_tensors,
), replace=True)
