"""A plain, slow implementation of the Vilazen decoder in float64 numpy: one function per mechanism, written from the
design's equations and sharing nothing with the engine.  It runs a whole sequence at once (no cache, no batching); the
engine's tests compare every way of cutting and batching against it.

The design in this file's notation.  T tokens, width D, rms(z) = z / sqrt(mean(z^2) + eps).

* stream: x = rms(E[tok]) (1 + w_0);
* layer: h = rms(x) (1 + w), x <- x + mixer(h) + B gelu(A h) (the feed-forward may be absent; gelu in its exact form);
* mixers: ``windowed_attention`` (type ``attention``), ``parallel`` (an attention with a sink beside a linear attention with
  a constant decay per head), ``latent_attention``;
* output: rms(x) (1 + w_f), logits = head x.
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


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu(z):
    """z times the standard normal distribution function at z."""
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def round_bf16(a):
    """Round float64 values to the nearest bfloat16 (ties to even), returned as float64."""
    f = np.asarray(a, dtype=np.float32)
    u = f.view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(a))


def _same(a):
    return a


# ------------------------------------------------------------------------------------------ rotation, softmax, masks
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


def visible(i, size=None, keep_first=0):
    """The positions that position i sees: the last ``size`` up to itself (None: all), and the first ``keep_first``."""
    j = np.arange(i + 1)
    return j if size is None else j[(i - j < size) | (j < keep_first)]


def attend(q, k, v, scale, size=None, keep_first=0, sinks=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; query head h uses key head h // (H / G)."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        see = visible(i, size, keep_first)
        for h in range(H):
            g = h // (H // G)
            s = (k[see, g] @ q[i, h]) * scale
            out[i, h] = softmax_with_sink(s, None if sinks is None else float(sinks[h])) @ v[see, g]
    return out


def gate_heads(o, z):
    """o [T, H, dv] times sigmoid(z) with z [T, H]."""
    return o * sigmoid(z)[:, :, None]


# ------------------------------------------------------------------------------------------ attention over a window
def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def windowed_attention(h, W, p, m, eps, rounder=_same, shared=None):
    """``shared`` (a dict that lives as long as the sequence): "v" is the values of the first layer that mixes."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    rot = m["rot"]
    q = rms(h @ W[p + "q"].T, eps) * W[p + "q.norm"]
    k = rms(h @ W[p + "k"].T, eps) * W[p + "k.norm"]
    q = rounder(rotate_neighbours(q.reshape(T, H, dk), pos, rot["dims"], rot["base"]))
    k = rounder(rotate_neighbours(k.reshape(T, G, dk), pos, rot["dims"], rot["base"]))
    v = h @ W[p + "v"].T
    if m.get("v_mix"):
        if "v" in shared:
            v = mix_values(v, shared["v"], float(W[p + "vmix"]))
        else:
            shared["v"] = v
    mask = m.get("mask") or {}
    o = attend(q, k, rounder(v).reshape(T, G, dv), m["scale"], mask.get("size"), mask.get("keep_first", 0))
    o = gate_heads(o, h @ W[p + "g"].T)
    return rounder(o.reshape(T, H * dv)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ two mixers side by side
def sink_attention(h, W, p, m, rounder=_same):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, rot = np.arange(T), m["rot"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(T, H, dk)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(T, G, dk)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).reshape(T, G, dv)
    q = rounder(rotate_neighbours(q, pos, rot["dims"], rot["base"]))
    k = rounder(rotate_neighbours(k, pos, rot["dims"], rot["base"]))
    o = attend(q, k, rounder(v), m["scale"], sinks=W[p + "sink"])
    o = gate_heads(o, h @ W[p + "g"].T)
    return rounder(o.reshape(T, H * dv)) @ W[p + "o"].T


def decay_scan(q, k, v, decay):
    """q, k [T, H, dk], v [T, H, dv], decay [H]: S_t = decay S_(t-1) + k_t v_t^T from S = 0, o_t = S_t^T q_t."""
    T, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    d = np.asarray(decay, dtype=np.float64)[:, None, None]
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out


def lightning_attention(h, W, p, m, eps, rounder=_same):
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[p + "q"].T).reshape(T, H, dk)
    k = silu(h @ W[p + "k"].T).reshape(T, H, dk)
    v = silu(h @ W[p + "v"].T).reshape(T, H, dv)
    o = decay_scan(q, k, v, m["decay"]).reshape(T, H * dv)
    o = rms(o, eps) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)
    return rounder(o) @ W[p + "o"].T


def parallel(h, W, p, m, eps, rounder=_same, shared=None):
    left = sink_attention(h, W, p + "left.", m["left"], rounder)
    right = lightning_attention(h, W, p + "right.", m["right"], eps, rounder)
    return m["left_scale"] * left + m["right_scale"] * right


# ------------------------------------------------------------------------------------------ latent attention
def latent_attention(h, W, p, m, eps, rounder=_same, shared=None):
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
        see = visible(i, (m.get("mask") or {}).get("size"))
        for hd in range(H):
            s = (k_plain[see, hd] @ q_plain[i, hd] + k_rot[see] @ q_rot[i, hd]) * m["scale"]
            out[i, hd] = softmax_with_sink(s) @ v[see, hd]
    return rounder(out.reshape(T, H * vd)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forward, layer, model
def dense(h, W, p, rounder=_same):
    return rounder(gelu(h @ W[p + "up"].T)) @ W[p + "down"].T


MIXERS = {"attention": windowed_attention, "parallel": parallel, "latent_attention": latent_attention}


def layer(x, W, cfg, index, rounder=_same, shared=None):
    L, eps, p = cfg["layers"][index], cfg["norm"]["eps"], f"l{index}."
    h = rounder(rms_around_zero(x, W[p + "norm1"], eps))
    out = x + MIXERS[L["type"]](h, W, p + "mix.", L["mixer"], eps, rounder, {} if shared is None else shared)
    if L.get("mlp") is not None:
        out = out + dense(h, W, p + "mlp.", rounder)
    return out


def forward(tokens, W, cfg, layer_outputs=None, rounded=False):
    """Logits [T, vocab] of a whole sequence; ``layer_outputs`` (a list) receives the stream after every layer.
    ``rounded``: everything a part hands to the next in 16 bits is rounded to bfloat16 (the yardstick of what 8-bit
    mantissas between the parts cost by themselves)."""
    rounder = round_bf16 if rounded else _same
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = rms_around_zero(W["embed"][list(tokens)], W["embed.norm"], eps)
    shared = {}
    for i in range(len(cfg["layers"])):
        x = layer(x, W, cfg, i, rounder, shared)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rounder(rms_around_zero(x, W["final.norm"], eps)) @ W["head"].T
