"""A plain, slow Gogotar: whole sequences, no cache, one function per mechanism.

Gogotar is a decoder of sandwich layers whose norms are layer norms without a bias, before and after each sublayer; a range of
layers may run several times in a row.  The mixer of a layer is `attention` (the values are the keys as projected; queries and
keys normed head by head, turned with frequencies stretched by wavelength, scores capped, every query confined to its own
chunk of positions) or `latent_attention` (queries, keys and values through low-rank latents, no positions); both put a learned
number per head into the softmax's denominator and gate their heads' outputs.  The feed-forward is dense (clamped, gated) or a
mixture of silu-gated experts weighed by a softmax over all experts.

This file shares no code with `kvad_b200`: it reads safetensors with its own few lines and computes with NumPy in float64,
with full score matrices.
"""
from __future__ import annotations

import json
import os
import struct

import numpy as np


def read_tensors(path):
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        blob = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw, dt = blob[lo:hi], info["dtype"]
        if dt == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif dt == "F32":
            a = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        else:
            raise ValueError(f"{name}: dtype {dt}")
        out[name] = a.reshape(info["shape"])
    return out


# ----------------------------------------------------------------------------- small pieces
def sigmoid(z):
    return np.where(z >= 0, 1.0, np.exp(-np.abs(z))) / (1.0 + np.exp(-np.abs(z)))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def capped(x, cap):
    """cap * tanh(x / cap); no cap: x."""
    return cap * np.tanh(x / cap) if cap else x


# ----------------------------------------------------------------------------- positions
def frequencies(rot):
    """One frequency per pair.  With `scaling` {factor, low, high, original}: pairs whose wavelength is below original / high keep
    theirs, those above original / low are slowed by `factor`, and between the two the one goes over into the other in
    proportion to original / wavelength."""
    f = np.array([float(rot["base"]) ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])
    sc = rot.get("scaling")
    if sc is None:
        return f
    out = np.empty_like(f)
    for i, fi in enumerate(f):
        length = 2.0 * np.pi / fi
        if length < sc["original"] / sc["high"]:
            out[i] = fi
        elif length > sc["original"] / sc["low"]:
            out[i] = fi / sc["factor"]
        else:
            s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
            out[i] = (1.0 - s) * fi / sc["factor"] + s * fi
    return out


def turn(x, pos, rot):
    """x [T, heads, dim]: entries i and i + dims/2 of the first `dims` turned by pos * frequency i; the rest passes."""
    n = rot["dims"] // 2
    a = np.asarray(pos, dtype=np.float64)[:, None, None] * frequencies(rot)
    u, v = x[..., :n], x[..., n:2 * n]
    out = x.copy()
    out[..., :n] = u * np.cos(a) - v * np.sin(a)
    out[..., n:2 * n] = v * np.cos(a) + u * np.sin(a)
    return out


# ----------------------------------------------------------------------------- attention
def chunk_mask(T, size):
    """[query, key]: no key after the query, none outside the query's chunk of `size` positions (None: no chunks)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i // size == j // size) if size else True)


def softmax_with_sink(s, sink):
    """Rows of scores (minus infinity: not seen) to weights; exp(sink) is one more term of the sum (None: it is not)."""
    m = s.max(-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    total = e.sum(-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - m)
    return e / total


def attend(q, k, v, scale, cap, sinks, mask):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // group
        s = np.where(mask, capped(q[:, h] @ k[:, g].T * scale, cap), -np.inf)
        out[:, h] = softmax_with_sink(s, None if sinks is None else sinks[h]) @ v[:, g]
    return out


def attention(h, w, p, m, eps):
    T, dk = h.shape[0], m["dim"]
    H, G = m["heads"], m.get("kv_heads") or m["heads"]
    q, k = (h @ w[p + "q"].T).reshape(T, H, dk), (h @ w[p + "k"].T).reshape(T, G, dk)
    v = k                                                    # the keys as projected
    pos = np.arange(T)
    q = turn(rms_norm(q, w[p + "q.norm"], eps), pos, m["rot"])
    k = turn(rms_norm(k, w[p + "k.norm"], eps), pos, m["rot"])
    o = attend(q, k, v, m["scale"], m.get("softcap"), w[p + "sink"], chunk_mask(T, m["mask"]["size"]))
    return (o * sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, H * dk) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, dk)
    c = rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
    k, v = (c @ w[p + "uk"].T).reshape(T, H, dk), (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = attend(q, k, v, m["scale"], None, w[p + "sink"], chunk_mask(T, None)).reshape(T, H * dv)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ----------------------------------------------------------------------------- feed-forwards
def clamped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w, p, limit):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def scores(z):
    e = np.exp(z - z.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def choose(z, top):
    """The `top` largest scores of every row (ties: the lower index) and those scores as they are."""
    s = scores(z)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, -1)


def moe_ff(h, w, p, mlp, margins=None, forced=None, own=None):
    """`forced` [T, top]: these experts instead of the router's own choice (their weights still from its scores);
    `own`, `margins`: lists that receive the router's own choice and by how much of a logit its last one was clear of the next."""
    z, top = h @ w[p + "router"].T, mlp["router"]["top"]
    chosen, weight = choose(z, top)
    if own is not None:
        own.append(chosen)
    if margins is not None:
        zs = np.sort(z, -1)[:, ::-1]
        margins.append(zs[:, top - 1] - zs[:, top] if top < z.shape[1] else np.full(z.shape[0], np.inf))
    if forced is not None:
        chosen = np.asarray(forced)
        weight = np.take_along_axis(scores(z), chosen, -1)
    out = np.zeros(h.shape)
    for e in range(mlp["router"]["experts"]):
        rows, slot = np.nonzero(chosen == e)
        if rows.size:
            out[rows] += weight[rows, slot][:, None] * expert(h[rows], w, f"{p}e{e}.")
    return out


# ----------------------------------------------------------------------------- the model
def run_order(config):
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward(config, w, tokens, return_layers=False, margins=None, forced=None, own=None):
    """Logits [T, vocab] of one whole sequence (and the stream after every layer that runs, if asked).  `forced`: per run of a
    routed layer, the experts [T, top] to use; `margins`, `own`: lists that receive, per such run, what its router chose by itself
    given the layers before it and how clearly."""
    forced = list(forced) if forced is not None else None
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    after = []
    for i in run_order(config):
        layer, p = config["layers"][i], f"l{i}."
        mixer = {"attention": attention, "latent_attention": latent_attention}[layer["type"]]
        x = x + layer_norm(mixer(layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps), w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = layer_norm(x, w[p + "norm2"], eps)
            y = dense_ff(h, w, p + "mlp.", mlp["limit"]) if mlp["kind"] == "dense" else \
                moe_ff(h, w, p + "mlp.", mlp, margins, forced.pop(0) if forced else None, own)
            x = x + layer_norm(y, w[p + "norm2b"], eps)
        after.append(x)
    logits = capped(layer_norm(x, w["final.norm"], eps) @ w["embed"].T, config.get("logit_softcap"))
    return (logits, np.stack(after)) if return_layers else logits


def greedy(config, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(config, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def load(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        config = json.load(f)
    return config, read_tensors(os.path.join(model_dir, "model.safetensors"))
