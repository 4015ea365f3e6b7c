"""A plain, slow implementation of the Zusotar decoder in float64 numpy: one function per mechanism, written from the
design's equations and sharing nothing with the engine.  It runs a whole sequence at once (no cache, no batching); the
engine's tests compare every way of cutting and batching against it.

The design in this file's notation.  T tokens, width D, rms(z) = z / sqrt(mean(z^2) + eps).

* embedding: X_0[t] = E[tok_t] + P[t], P a learned row per position;
* layer i, on its input x: y = x + m rms(mixer(rms(x) (1 + a))) (1 + b), X_(i+1) = y + m rms(ff(rms(y) (1 + c))) (1 + d),
  all four norms' weights stored around zero; the feed-forward with its two norms may be absent;
* depth average: what layer i hands on is sum_j w_i[j] X_j over j = 0 .. i + 1 (the embedding output and the layers'
  results, none of them averaged);
* mixers: ``latent_attention``, ``log_bias_attention`` (type ``attention``), ``gated_linear_attention`` (type ``gla``);
* feed-forward: ``gated`` (dense) or ``expert_mixture``;
* output: rms(x) (1 + w), logits = head x.
"""
from __future__ import annotations

import math

import numpy as np


def rms(z, eps):
    return z / np.sqrt((z * z).mean(-1, keepdims=True) + eps)


def rms_around_zero(z, w, eps):
    """The model's norm: the stored weight is the distance from 1."""
    return rms(z, eps) * (1.0 + w)


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def silu(z):
    return z * sigmoid(z)


def round_bf16(a):
    """Round float64 values to the nearest bfloat16 (ties to even), returned as float64."""
    f = np.asarray(a, dtype=np.float32)
    u = f.view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(a))


def _same(a):
    return a


# ------------------------------------------------------------------------------------------ embedding, depth average
def embedding(tokens, W):
    return W["embed"][list(tokens)] + W["pos"][:len(tokens)]


def depth_average(results, weights):
    """sum_j weights[j] results[j]; ``results``: the embedding output, then every layer's result so far."""
    assert len(results) == len(weights)
    out = np.zeros_like(results[0])
    for r, w in zip(results, weights):
        out += w * r
    return out


# ------------------------------------------------------------------------------------------ latent attention
def rotate_neighbours(v, positions, dims, base):
    """v [T, ..., n]: channels 2i and 2i+1 of the first ``dims`` turn together by position * base^(-2i / dims)."""
    out = v.copy()
    f = float(base) ** (-2.0 * np.arange(dims // 2) / dims)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    shape = (len(positions),) + (1,) * (v.ndim - 2) + (dims // 2,)
    c, s = np.cos(ang).reshape(shape), np.sin(ang).reshape(shape)
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def softmax_with_sink(s, sink=None):
    """Weights of the scores s [keys]; with ``sink`` the denominator has the extra term exp(sink)."""
    top = s.max() if sink is None else max(s.max(), sink)
    e = np.exp(s - top)
    return e / (e.sum() + (math.exp(sink - top) if sink is not None else 0.0))


def latent_attention(h, W, p, m, eps, rounder=_same):
    T = h.shape[0]
    H, dim, rd, vd, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (h @ W[p + "q"].T).reshape(T, H, dim + rd)
    q_plain = rounder(q[..., :dim])
    q_rot = rounder(rotate_neighbours(q[..., dim:], pos, m["rot"]["dims"], m["rot"]["base"]))
    d = h @ W[p + "dkv"].T
    c = rounder(rms(d[:, :r], eps) * W[p + "dkv.norm"])
    k_rot = rounder(rotate_neighbours(d[:, r:], pos, m["rot"]["dims"], m["rot"]["base"]))
    k_plain = rounder((c @ W[p + "uk"].T).reshape(T, H, dim))
    v = rounder((c @ W[p + "uv"].T).reshape(T, H, vd))
    out = np.zeros((T, H, vd))
    for i in range(T):
        for hd in range(H):
            s = (k_plain[:i + 1, hd] @ q_plain[i, hd] + k_rot[:i + 1] @ q_rot[i, hd]) * m["scale"]
            out[i, hd] = softmax_with_sink(s, float(W[p + "sink"][hd])) @ v[:i + 1, hd]
    return rounder(out.reshape(T, H * vd)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ window attention
def attend_log_bias(q, k, v, window, scale, r1, r2):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv]: row i sees the positions j with 0 <= i - j < window; the score is
    (q . k) scale - r1[h] ln(1 + r2[h] (i - j)); ordinary softmax.  Returns [T, H, dv]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = max(0, i - window + 1)
        dist = i - np.arange(lo, i + 1)
        for hd in range(H):
            g = hd // (H // G)
            s = (k[lo:i + 1, g] @ q[i, hd]) * scale - r1[hd] * np.log1p(r2[hd] * dist)
            out[i, hd] = softmax_with_sink(s) @ v[lo:i + 1, g]
    return out


def log_bias_attention(h, W, p, m, eps, rounder=_same):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rounder((h @ W[p + "q"].T).reshape(T, H, dk))
    k = rounder((h @ W[p + "k"].T).reshape(T, G, dk))
    v = rounder(rms((h @ W[p + "v"].T).reshape(T, G, dv), eps))
    out = attend_log_bias(q, k, v, m["mask"]["size"], m["scale"], W[p + "r1"], W[p + "r2"])
    return rounder(out.reshape(T, H * dv) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ gated linear attention
def linear_attention_scan(q, k, v, log_decay):
    """q, k, log_decay [T, H, dk], v [T, H, dv]: S_t = diag(exp(log_decay_t)) S_(t-1) + k_t v_t^T from S = 0,
    o_t = S_t^T q_t.  Returns [T, H, dv]."""
    T, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = np.exp(log_decay[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out


def gated_linear_attention(h, W, p, m, eps, rounder=_same):
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, dk)
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    log_decay = -np.logaddexp(0.0, -z).reshape(T, H, dk) / m["tau"]              # ln of sigmoid(z)^(1 / tau)
    o = rms(linear_attention_scan(q, k, v, log_decay), eps) * W[p + "norm"]
    return rounder(o.reshape(T, H * dv) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forward
def gated(h, W, p, rounder=_same):
    return rounder(silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W, p, router):
    """(chosen experts [T, top], weights [T, top]): the largest sigmoid scores among the experts of the best groups (a
    group's score: the sum of its two largest scores); the weights are the scores themselves."""
    n, top = router["experts"], router["top"]
    s = sigmoid(h @ W[p + "router"].T)
    choice = s
    groups = router.get("groups")
    if groups is not None:
        per = n // groups["count"]
        best = np.sort(s.reshape(-1, groups["count"], per), axis=-1)[..., -2:].sum(-1)
        kept = np.argsort(-best, axis=-1, kind="stable")[:, :groups["keep"]]
        allowed = np.zeros(best.shape, dtype=bool)
        np.put_along_axis(allowed, kept, True, axis=-1)
        choice = np.where(np.repeat(allowed, per, axis=-1), s, -np.inf)
    ids = np.argsort(-choice, axis=-1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=-1)


def route_margin(h, W, p, router):
    """How close the router's choices are, per token: the smaller of the gaps between the last chosen and the first refused
    score, and between the last kept and the first refused group (infinite where there is nothing to refuse)."""
    s = sigmoid(h @ W[p + "router"].T)
    T, n = s.shape
    gap, allowed = np.full(T, np.inf), np.ones((T, n), dtype=bool)
    groups = router.get("groups")
    if groups is not None and groups["keep"] < groups["count"]:
        per, keep = n // groups["count"], groups["keep"]
        best = np.sort(s.reshape(T, groups["count"], per), axis=-1)[..., -2:].sum(-1)
        order = np.sort(best, axis=-1)[:, ::-1]
        gap = order[:, keep - 1] - order[:, keep]
        allowed = np.repeat(best >= order[:, keep - 1:keep], per, axis=-1)
    for t in range(T):
        order = np.sort(s[t, allowed[t]])[::-1]
        if router["top"] < len(order):
            gap[t] = min(gap[t], order[router["top"] - 1] - order[router["top"]])
    return gap


def expert_mixture(h, W, p, mlp, rounder=_same, margins=None):
    if margins is not None:
        margins.append(route_margin(h, W, p, mlp["router"]))
    ids, weights = route(h, W, p, mlp["router"])
    out = np.zeros(h.shape)
    for t in range(h.shape[0]):
        for e, w in zip(ids[t], weights[t]):
            out[t] += w * gated(h[t:t + 1], W, f"{p}e{int(e)}.", rounder)[0]
    if mlp.get("shared") is not None:
        out += gated(h, W, p + "shared.", rounder)
    return out


# ------------------------------------------------------------------------------------------ layer, model
MIXERS = {"latent_attention": latent_attention, "attention": log_bias_attention, "gla": gated_linear_attention}


def layer(x, W, cfg, index, rounder=_same, margins=None):
    """The layer's result, before the depth average."""
    L, eps, m, p = cfg["layers"][index], cfg["norm"]["eps"], cfg["residual_mult"], f"l{index}."
    y = MIXERS[L["type"]](rounder(rms_around_zero(x, W[p + "norm1"], eps)), W, p + "mix.", L["mixer"], eps, rounder)
    x = x + m * rms_around_zero(y, W[p + "norm1b"], eps)
    mlp = L.get("mlp")
    if mlp is not None:
        h = rounder(rms_around_zero(x, W[p + "norm2"], eps))
        y = gated(h, W, p + "mlp.", rounder) if mlp["kind"] == "dense" else expert_mixture(h, W, p + "mlp.", mlp, rounder, margins)
        x = x + m * rms_around_zero(y, W[p + "norm2b"], eps)
    return x


def forward(tokens, W, cfg, layer_outputs=None, rounded=False, margins=None):
    """Logits [T, vocab] of a whole sequence; ``layer_outputs`` (a list) receives what every layer hands on, ``margins`` (a
    list) how close every router's choices are.
    ``rounded``: everything a part hands to the next in 16 bits is rounded to bfloat16 (the yardstick of what 8-bit
    mantissas between the parts cost by themselves)."""
    rounder = round_bf16 if rounded else _same
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    x = embedding(tokens, W)
    results = [x]
    for i in range(len(cfg["layers"])):
        results.append(layer(x, W, cfg, i, rounder, margins))
        x = depth_average(results, W[f"l{i}.dwa"])
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rounder(rms_around_zero(x, W["final.norm"], cfg["norm"]["eps"])) @ W["head"].T
