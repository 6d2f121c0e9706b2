"""Tugolix: a decoder whose residual stream is several copies side by side, mixed at every sublayer (hyper-connections).

    x_1 = .. = x_n = embed[token]
    per layer, for the mixer and then for the feed-forward (which may be absent):
        y = sublayer(norm(sum_s in[s] x_s));   x_t <- sum_s mix[s, t] x_s + out[t] y
    logits = head . norm(sum_s x_s) * logit_scale

Norms are layer norms with weight and bias.  The mixer of a layer is one of `gla` (linear attention with a decay per key
channel, sigmoid(z)^(1 / tau), a norm per head and a silu gate), `latent_attention` (keys and values through one low-rank latent,
no positions; with `kv_from`: j the layer keeps nothing and reads layer j's cached latent) and `channel_delta` (the delta rule
with a decay per key channel, short causal convolutions on q, k and v).  The feed-forward is `dense` (down(silu(gate h) * (up h)),
biases) or `moe`: clamped experts chosen by sigmoid scores plus a correction within the best groups of experts, weighing their
scores over the chosen scores' sum times a constant.

config.json: `architecture`, `vocab`, `width`, `streams`, `logit_scale` (absent: 1), `norm.eps` and `layers`, a list of {`type`,
`mixer`, `mlp`}.  `gla`: `heads`, `dim`, `vdim`, `tau`.  `latent_attention`: `heads`, `dim`, `vdim`, `kv_rank`, `scale`, `kv_from`
(absent: a latent of its own).  `channel_delta`: `heads`, `kv_heads`, `dim`, `vdim`, `conv`.  `mlp`: null, {`kind`: "dense", `ff`}
or {`kind`: "moe", `router`: {`experts`, `top`, `scale`, `groups`: {`count`, `keep`}}, `expert`: {`ff`, `limit`}}.  Tensors: `embed`,
`l<i>.norm1|norm2` (`.b`), `l<i>.hc1|hc2.in|out|mix`, `l<i>.mix.<name>`, `l<i>.mlp.<name>`, `final.norm` (`.b`), `head`; matrices are
`[out, in]`.  The ranks of the low-rank maps (`a1`, `g1`) are read from the tensors' shapes when a model folder is loaded and
stand in the typed configuration as `mixer.decay_rank` / `mixer.gate_rank`.  This module only describes: the configuration, the
plan (which parts, with which sizes and tensor names) and the random-weights recipe; all computing is in the parts.
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass, replace

from ..config.json_view import ConfigError, JsonView
from ..config.registry import Architecture, register
from ..parts.base import PartSpec
from .plan import LayerCall, ModelPlan

MIXER_TYPES = ("gla", "latent_attention", "channel_delta")
#: constants the design fixes
EXPERT_ALPHA = 1.702        # the experts' gate is g * sigmoid(EXPERT_ALPHA * g)
UNIT_EPS = 1e-6             # under the root that makes the delta rule's q and k unit vectors
DEFAULT_RANK = 20           # random-weights mode: rank of the low-rank maps where a configuration names none
MAX_STREAMS, MAX_GROUPS = 16, 256


@dataclass(frozen=True)
class TugolixConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    logit_scale: float
    layers: tuple            # of dicts {"type", "mixer", "mlp"} as config.json has them
    arch_id: str = "tugolix"


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
    v = float(_need(d, key, where))
    if not v > 0:
        raise ConfigError(f"config: {where}: `{key}` must be positive")
    return v


def _groups(router: dict) -> tuple:
    g = router.get("groups")
    return (1, 1) if g is None else (g["count"], g["keep"])


def _check_mixer(layers: list, i: int, where: str) -> None:
    layer = layers[i]
    m = layer.get("mixer")
    if not isinstance(m, dict):
        raise ConfigError(f"config: {where} has no `mixer`")
    heads = _pos_int(m, "heads", where)
    _pos_int(m, "dim", where), _pos_int(m, "vdim", where)
    if layer["type"] == "gla":
        _positive(m, "tau", where)
    elif layer["type"] == "channel_delta":
        kv = _pos_int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads      # (absent: a query/key head per head)
        if heads % kv:
            raise ConfigError(f"config: {where}: {heads} heads do not divide into {kv} query/key heads")
        _pos_int(m, "conv", where)
    else:
        rank = _pos_int(m, "kv_rank", where)
        _need(m, "scale", where)
        src = m.get("kv_from")
        if src is None:
            return
        if isinstance(src, bool) or not isinstance(src, int) or not (0 <= src < i):
            raise ConfigError(f"config: {where}: `kv_from` must name an earlier layer")
        if layers[src]["type"] != "latent_attention" or layers[src]["mixer"].get("kv_from") is not None:
            raise ConfigError(f"config: {where}: `kv_from` must name a latent-attention layer with a latent of its own")
        if layers[src]["mixer"]["kv_rank"] != rank:
            raise ConfigError(f"config: {where}: the layer it reads from must have its latent size")


def _check_mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config: {where}: `mlp` is null or of kind `dense` or `moe`")
    if mlp["kind"] == "dense":
        _pos_int(mlp, "ff", where + " mlp")
        return
    r, where_r = mlp.get("router"), where + " router"
    experts, top = _pos_int(r, "experts", where_r), _pos_int(r, "top", where_r)
    _positive(r, "scale", where_r)
    count, keep = 1, 1
    if r.get("groups") is not None:
        count, keep = _pos_int(r["groups"], "count", where_r + " groups"), _pos_int(r["groups"], "keep", where_r + " groups")
    if keep > count or experts % count or count > MAX_GROUPS:
        raise ConfigError(f"config: {where_r}: {experts} experts do not form {count} equal groups (at most {MAX_GROUPS}) of which {keep} are kept")
    if top > keep * (experts // count):
        raise ConfigError(f"config: {where_r}: more experts a token than can be chosen from")
    _pos_int(mlp.get("expert"), "ff", where + " expert"), _positive(mlp.get("expert"), "limit", where + " expert")


def read_config(view: JsonView) -> TugolixConfig:
    tree = view.tree
    vocab, width, streams = (_pos_int(tree, k, "the model") for k in ("vocab", "width", "streams"))
    if streams > MAX_STREAMS:
        raise ConfigError(f"config: at most {MAX_STREAMS} `streams`")
    eps = float(_need(tree.get("norm"), "eps", "`norm`"))
    logit_scale = 1.0 if tree.get("logit_scale") is None else float(_need(tree, "logit_scale", "the model"))
    layers = tree.get("layers")
    if not isinstance(layers, list) or not layers:
        raise ConfigError("config: `layers` must be a non-empty list")
    for i, layer in enumerate(layers):
        where = f"layer {i}"
        if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
            raise ConfigError(f"config: {where}: `type` must be one of {MIXER_TYPES}")
        _check_mixer(layers, i, where)
        _check_mlp(layer.get("mlp"), where)
    return TugolixConfig(vocab=vocab, width=width, streams=streams, norm_eps=eps, logit_scale=logit_scale, layers=tuple(copy.deepcopy(layers)))


def with_checkpoint_shapes(c: TugolixConfig, shape_of) -> TugolixConfig:
    """Sizes that only the tensors' shapes give: the ranks of the low-rank maps."""
    layers = copy.deepcopy(list(c.layers))
    names = {"gla": (("decay_rank", "a1"),), "channel_delta": (("decay_rank", "a1"), ("gate_rank", "g1")), "latent_attention": ()}
    for i, layer in enumerate(layers):
        for key, name in names[layer["type"]]:
            shape = shape_of(f"l{i}.mix.{name}")
            if shape is not None and len(shape) == 2:
                layer["mixer"][key] = int(shape[0])
    return replace(c, layers=tuple(layers))


def write_config(c: TugolixConfig) -> dict:
    layers = copy.deepcopy(list(c.layers))
    for layer in layers:                      # (the ranks live in the tensors' shapes, not in config.json)
        layer["mixer"].pop("decay_rank", None), layer["mixer"].pop("gate_rank", None)
    return {"architecture": "Tugolix", "vocab": c.vocab, "width": c.width, "streams": c.streams, "norm": {"eps": c.norm_eps},
            "logit_scale": c.logit_scale, "layers": layers}


def _mixer_spec(c: TugolixConfig, layer: dict) -> PartSpec:
    m, kind = layer["mixer"], layer["type"]
    sizes = {"width": c.width, "n_heads": m["heads"], "value_dim": m["vdim"], "norm_eps": c.norm_eps}
    if kind == "gla":
        return PartSpec("gated_linear_attention", {**sizes, "key_dim": m["dim"], "tau": m["tau"], "decay_rank": m.get("decay_rank", DEFAULT_RANK)})
    if kind == "channel_delta":
        return PartSpec("gated_delta_rule", {
            **sizes, "n_kv_heads": m.get("kv_heads") or m["heads"], "key_dim": m["dim"], "conv_taps": m["conv"], "unit_eps": UNIT_EPS,
            "decay_rank": m.get("decay_rank", DEFAULT_RANK), "gate_rank": m.get("gate_rank", DEFAULT_RANK)})
    return PartSpec("latent_attention", {**sizes, "nope_dim": m["dim"], "rot_dim": 0, "q_rank": None, "kv_rank": m["kv_rank"],
                                         "score_scale": m["scale"], "own_kv": m.get("kv_from") is None})


def _mlp_spec(c: TugolixConfig, mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("gated_mlp", {"width": c.width, "hidden": mlp["ff"], "activation": "silu", "bias_suffix": ".b"})
    r = mlp["router"]
    return PartSpec("routed_mlp", {
        "width": c.width, "n_experts": r["experts"], "top": r["top"], "hidden": mlp["expert"]["ff"], "limit": mlp["expert"]["limit"],
        "alpha": EXPERT_ALPHA, "routing": {"groups": _groups(r), "scale": r["scale"]}})


def plan(c: TugolixConfig) -> ModelPlan:
    norm = PartSpec("layernorm", {"width": c.width, "eps": c.norm_eps, "name": "", "bias_name": ".b"})
    blocks, prefixes, order, kinds = [], [], [], []
    for i, layer in enumerate(c.layers):
        blocks.append(PartSpec("hyper_connections", {"streams": c.streams, "norm": norm, "mixer": _mixer_spec(c, layer),
                                                     "feed_forward": _mlp_spec(c, layer.get("mlp"))}))
        prefixes.append(f"l{i}.")
        src = layer["mixer"].get("kv_from") if layer["type"] == "latent_attention" else None
        order.append(LayerCall(i, i) if src is None else LayerCall(i, int(src), writes_cache=False))
        kinds.append({"gla": "g", "latent_attention": "l", "channel_delta": "d"}[layer["type"]])
    return ModelPlan(
        arch_id="tugolix", vocab_size=c.vocab, width=c.width,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "width": c.width, "name": "embed"}),
        blocks=tuple(blocks), block_prefixes=tuple(prefixes),
        head=PartSpec("lm_head", {"vocab_size": c.vocab, "width": c.width, "norm": norm, "tied": False, "bias": False,
                                  "norm_name": "final.norm", "name": "head", "weight_name": "", "logit_scale": c.logit_scale}),
        order=tuple(order), max_positions=None,
        summary=f"tugolix · {len(c.layers)} layers ({''.join(kinds)}) · {c.streams} x {c.width} wide · {c.vocab} vocab",
    )


def random_tensors(c: TugolixConfig, rng) -> dict:
    """Matrices ~N(0, 1/in), the embedding ~N(0, 1), norm weights near 1 and their biases away from 0, the copies' mixes near
    the identity, decays spread so that some channels forget at once and some hardly, corrections of the order of the scores'
    differences."""
    def mat(out, inp, gain=1.0):
        return rng.normal((out, inp), gain / math.sqrt(inp))

    def norm(t, name):
        t[name], t[name + ".b"] = rng.normal((w,), 0.1, 1.0), rng.normal((w,), 0.1)

    w, n = c.width, c.streams
    t = {"embed": rng.normal((c.vocab, w), 1.0), "head": mat(c.vocab, w, 2.0)}
    norm(t, "final.norm")
    for i, layer in enumerate(c.layers):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        for q in (1, 2) if mlp is not None else (1,):
            norm(t, p + f"norm{q}")
            t[p + f"hc{q}.in"], t[p + f"hc{q}.out"] = rng.normal((n,), 0.3, 1.0 / n), rng.normal((n,), 0.2, 0.6)
            mix = rng.normal((n, n), 0.15)
            mix.diagonal().add_(0.9)
            t[p + f"hc{q}.mix"] = mix
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "gla":
            ra = m.get("decay_rank", DEFAULT_RANK)
            t[p + "mix.q"], t[p + "mix.k"], t[p + "mix.v"] = mat(H * dk, w, 2.0), mat(H * dk, w), mat(H * dv, w)
            t[p + "mix.a1"], t[p + "mix.a2"], t[p + "mix.a2.b"] = mat(ra, w), mat(H * dk, ra, 2.0), rng.normal((H * dk,), 2.0, 1.0)
            t[p + "mix.g"], t[p + "mix.norm"], t[p + "mix.o"] = mat(H * dv, w), rng.normal((dv,), 0.1, 1.0), mat(w, H * dv)
        elif layer["type"] == "channel_delta":
            G, taps = m.get("kv_heads") or H, m["conv"]
            ra, rg = m.get("decay_rank", DEFAULT_RANK), m.get("gate_rank", DEFAULT_RANK)
            for name, ch in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                t[p + f"mix.{name}"], t[p + f"mix.{name}.conv"] = mat(ch, w, 2.0), rng.normal((ch, taps), 0.5)
            t[p + "mix.b"], t[p + "mix.A_log"] = mat(H, w, 2.0), rng.normal((H,), 0.5, -1.0)
            t[p + "mix.a1"], t[p + "mix.a2"], t[p + "mix.dt_bias"] = mat(ra, w), mat(H * dk, ra, 2.0), rng.normal((H * dk,), 1.0, -1.0)
            t[p + "mix.g1"], t[p + "mix.g2"] = mat(rg, w), mat(H * dv, rg, 2.0)
            t[p + "mix.norm"], t[p + "mix.o"] = rng.normal((dv,), 0.1, 1.0), mat(w, H * dv)
        else:
            rk = m["kv_rank"]
            t[p + "mix.q"] = mat(H * dk, w, 2.0)
            if m.get("kv_from") is None:
                t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = mat(rk, w), rng.normal((rk,), 0.1, 1.0)
            t[p + "mix.uk"], t[p + "mix.uv"], t[p + "mix.o"] = mat(H * dk, rk, 2.0), mat(H * dv, rk), mat(w, H * dv)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            for name, out, inp in (("gate", mlp["ff"], w), ("up", mlp["ff"], w), ("down", w, mlp["ff"])):
                t[p + "mlp." + name], t[p + f"mlp.{name}.b"] = mat(out, inp), rng.normal((out,), 0.2)
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        for e in range(E):
            t[p + f"mlp.e{e}.gate"], t[p + f"mlp.e{e}.up"], t[p + f"mlp.e{e}.down"] = mat(ff, w, 2.0), mat(ff, w, 2.0), mat(w, ff)
        t[p + "mlp.router"], t[p + "mlp.correction"] = mat(E, w, 3.0), rng.normal((E,), 0.2)
    return t


ARCH = register(Architecture(
    id="tugolix", model_types=("tugolix",),
    about="Tugolix: several copies of the stream mixed at every sublayer; gated linear attention, latent attention without positions or delta rule; dense or group-routed feed-forward",
    read_config=read_config, plan=plan, write_config=write_config, random_tensors=random_tensors,
    with_checkpoint_shapes=with_checkpoint_shapes,
), replace=True)
