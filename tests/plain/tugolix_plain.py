"""A plain, slow Tugolix: whole sequences, no cache, one function per mechanism.

Tugolix is a decoder whose residual stream is several copies side by side.  Every sublayer reads one weighted sum of
the copies through a layer norm; afterwards all copies are mixed with one another and each takes its share of the
sublayer's result.  The mixer of a layer is one of `gla` (linear attention with a decay per key channel), `latent_attention`
(keys and values rebuilt from one low-rank latent, no positions; a layer may read another layer's latent) and
`channel_delta` (the delta rule with a decay per key channel and short causal convolutions).  The feed-forward is dense
(gated, silu, biases) or a mixture of clamped experts chosen group by group from sigmoid scores.

This file shares no code with `kvad_b200`: it reads safetensors with its own few lines and computes with NumPy in
float64, token by token where the design has a recurrence and with full score matrices where it has attention.
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


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w + b


def softmax_rows(s):
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


# ----------------------------------------------------------------------------- several copies of the stream
def read_streams(xs, weights):
    """What a sublayer sees: xs [copies, T, width], weights [copies] -> [T, width]."""
    return sum(weights[s] * xs[s] for s in range(len(weights)))


def write_streams(xs, mix, share, y):
    """All copies at once from the old ones: copy t becomes sum_s mix[s, t] x_s + share[t] y."""
    n = len(share)
    return np.stack([sum(mix[s, t] * xs[s] for s in range(n)) + share[t] * y for t in range(n)])


# ----------------------------------------------------------------------------- mixers
def gla_decay(z, tau):
    return sigmoid(z) ** (1.0 / tau)


def gla_cell(q, k, v, alpha, S=None):
    """One head, token by token: q, k, alpha [T, dk], v [T, dv].  Returns (read-outs [T, dv], S [dk, dv])."""
    S = np.zeros((q.shape[1], v.shape[1])) if S is None else S
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        S = alpha[t][:, None] * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def gla(h, w, p, m, eps):
    """Gated linear attention.  h [T, width]; returns [T, width]."""
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, dk)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    alpha = gla_decay(((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]).reshape(T, H, dk), m["tau"])
    out = np.stack([gla_cell(q[:, a], k[:, a], v[:, a], alpha[:, a])[0] for a in range(H)], axis=1)
    o = (rms_unit(out, eps) * w[p + "norm"][None, None, :]).reshape(T, H * dv) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def latent(h, w, p, eps):
    """What a latent layer keeps per position."""
    return rms_unit(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]


def latent_attention(h, w, p, m, c):
    """Softmax attention with keys and values rebuilt head by head from the kept latent c [T, kv_rank]."""
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, dk)
    k = (c @ w[p + "uk"].T).reshape(T, H, dk)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    mask = np.tril(np.ones((T, T), dtype=bool))
    out = np.zeros((T, H, dv))
    for a in range(H):
        out[:, a] = softmax_rows(np.where(mask, q[:, a] @ k[:, a].T * m["scale"], -np.inf)) @ v[:, a]
    return out.reshape(T, H * dv) @ w[p + "o"].T


def short_conv(x, taps):
    """Causal convolution over time per channel: x [T, C], taps [C, n], the last column meets the current row."""
    T, n = x.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x], axis=0)
    return sum(padded[j:j + T] * taps[:, j][None, :] for j in range(n))


def unit_vectors(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_cell(q, k, v, beta, g, S=None):
    """One head, token by token: q, k, g [T, dk], v [T, dv], beta [T].  Returns (read-outs [T, dv], S [dk, dv])."""
    S = np.zeros((q.shape[1], v.shape[1])) if S is None else S
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out, S


def channel_delta(h, w, p, m, eps):
    """The delta rule with a decay per key channel."""
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    q = silu(short_conv(h @ w[p + "q"].T, w[p + "q.conv"])).reshape(T, G, dk)
    k = silu(short_conv(h @ w[p + "k"].T, w[p + "k.conv"])).reshape(T, G, dk)
    v = silu(short_conv(h @ w[p + "v"].T, w[p + "v.conv"])).reshape(T, H, dv)
    q, k = unit_vectors(q) * dk ** -0.5, unit_vectors(k)
    beta = sigmoid(h @ w[p + "b"].T)
    a = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, dk)
    g = np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(a))
    out = np.stack([delta_cell(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], g[:, a])[0] for a in range(H)], axis=1)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, dv)
    return (rms_unit(out, eps) * w[p + "norm"][None, None, :] * gate).reshape(T, H * dv) @ w[p + "o"].T


# ----------------------------------------------------------------------------- feed-forwards
def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T + w[p + "gate.b"]) * (h @ w[p + "up"].T + w[p + "up.b"])) @ w[p + "down"].T + w[p + "down.b"]


def clamped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def clamped_expert(h, w, p, limit):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def open_choices(z, correction, groups):
    """Choice scores with the experts of groups that are not among the best set to minus infinity, and the groups' own
    scores [T, groups] (ties: the lower index)."""
    c = sigmoid(z) + correction
    T, E = c.shape
    n, keep = groups["count"], groups["keep"]
    per = E // n
    gs = np.sort(c.reshape(T, n, per), axis=-1)[..., -2:].sum(-1)
    kept = np.argsort(-gs, axis=-1, kind="stable")[:, :keep]
    allowed = np.zeros((T, n), dtype=bool)
    np.put_along_axis(allowed, kept, True, -1)
    return np.where(np.repeat(allowed, per, axis=-1), c, -np.inf), gs


def weigh(z, chosen, scale):
    s = np.take_along_axis(sigmoid(z), chosen, -1)
    return s / (s.sum(-1, keepdims=True) + 1e-20) * scale


def choose(z, correction, router):
    """(chosen experts [T, top], their weights [T, top])."""
    c, _ = open_choices(z, correction, router["groups"])
    chosen = np.argsort(-c, axis=-1, kind="stable")[:, :router["top"]]
    return chosen, weigh(z, chosen, router["scale"])


def routing_margin(z, correction, router):
    """Per row, by how much the choice is clear: of the last kept group over the next one, and of the last chosen expert over
    the next one that could be chosen."""
    c, gs = open_choices(z, correction, router["groups"])
    n, keep, top = router["groups"]["count"], router["groups"]["keep"], router["top"]
    margin = np.full(z.shape[0], np.inf)
    if keep < n:
        g = np.sort(gs, -1)[:, ::-1]
        margin = np.minimum(margin, g[:, keep - 1] - g[:, keep])
    if top < keep * (z.shape[1] // n):
        e = np.sort(c, -1)[:, ::-1]
        margin = np.minimum(margin, e[:, top - 1] - e[:, top])
    return margin


def moe_ff(h, w, p, mlp, margins=None, forced=None, own=None):
    """`forced` [T, top]: these experts instead of the router's own choice (their weights still from its scores);
    `own`, `margins`: lists that receive the router's own choice and its margins."""
    z, router = h @ w[p + "router"].T, mlp["router"]
    chosen, weight = choose(z, w[p + "correction"], router)
    if own is not None:
        own.append(chosen)
    if margins is not None:
        margins.append(routing_margin(z, w[p + "correction"], router))
    if forced is not None:
        chosen = np.asarray(forced)
        weight = weigh(z, chosen, router["scale"])
    out = np.zeros((h.shape[0], w[p + "e0.down"].shape[0]))
    for e in range(router["experts"]):
        rows, slot = np.nonzero(chosen == e)
        if rows.size:
            out[rows] += weight[rows, slot][:, None] * clamped_expert(h[rows], w, f"{p}e{e}.", mlp["expert"]["limit"])
    return out


# ----------------------------------------------------------------------------- the model
def forward(config, w, tokens, return_layers=False, margins=None, forced=None, own=None):
    """Logits [T, vocab] of one whole sequence (and the sum of the streams after every layer, if asked).  `forced`: per
    routed layer, the experts [T, top] to use; `margins`, `own`: lists that receive, per routed layer, what its router
    chose by itself given the layers before it and how clearly."""
    forced = list(forced) if forced is not None else None
    eps = config["norm"]["eps"]
    xs = np.stack([w["embed"][np.asarray(tokens)]] * config["streams"])
    kept, after = {}, []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = layer_norm(read_streams(xs, w[p + "hc1.in"]), w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer["type"] == "gla":
            y = gla(h, w, p + "mix.", m, eps)
        elif layer["type"] == "channel_delta":
            y = channel_delta(h, w, p + "mix.", m, eps)
        elif layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                src = i
                kept[i] = latent(h, w, p + "mix.", eps)
            y = latent_attention(h, w, p + "mix.", m, kept[src])
        else:
            raise ValueError(layer["type"])
        xs = write_streams(xs, w[p + "hc1.mix"], w[p + "hc1.out"], y)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = layer_norm(read_streams(xs, w[p + "hc2.in"]), w[p + "norm2"], w[p + "norm2.b"], eps)
            y = dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp, margins, forced.pop(0) if forced else None, own)
            xs = write_streams(xs, w[p + "hc2.mix"], w[p + "hc2.out"], y)
        after.append(xs.sum(0))
    logits = layer_norm(xs.sum(0), w["final.norm"], w["final.norm.b"], eps) @ w["head"].T * config["logit_scale"]
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
