"""Plain, slow Kitonex in numpy: the oracle the engine is compared with.

Whole sequences, no cache, no batching, float64, one function per mechanism, query by query, written from the design's
equations; it shares no code with the package (only the file readers of the other oracle).

    input:   e = E[token] + P[position];  S copies x_1 .. x_S = e
    sublayer q (1: mixer, 2: feed-forward; a layer may end after the first):
             u = sum_s in[s] x_s;   y = sublayer(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y     (all t at once)
    norm:    v / sqrt(mean(v^2) + eps) * w
    output:  W_head norm(sum_s x_s)
"""
from __future__ import annotations

import math
import os

import numpy as np

from plain_gemma2 import read_config, read_safetensors  # noqa: F401  (file formats only)


def load_folder(folder):
    w = read_safetensors(os.path.join(folder, "model.safetensors"))
    return read_config(folder), {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def short_conv(u, weight):
    """y_t[c] = sum_j weight[c, j] u_(t - (K - 1) + j)[c], zeros before the first row."""
    T, K = u.shape[0], weight.shape[1]
    y = np.zeros_like(u)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += weight[:, j] * u[s]
    return y


def bucket(n, buckets, largest):
    """Distances below B/2 have a bucket of their own; larger ones share buckets that widen as the logarithm up to `largest`."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(largest / half) * (buckets - half)))


def first_visible(i, size):
    """Chunks of `size` positions counted from 0: the first position of the chunk that position i lies in."""
    return 0 if size is None else (i // size) * size


def attend(q, k, v, scale, rel, largest, size):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]: softmax with one added to the denominator over the visible keys of
    scale * (q . k) + rel[bucket(distance), head]."""
    T, H, _ = q.shape
    G = k.shape[1]
    B = rel.shape[0]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = first_visible(i, size)
        b = [bucket(i - j, B, largest) for j in range(lo, i + 1)]
        for a in range(H):
            g = a // (H // G)
            s = k[lo:i + 1, g] @ q[i, a] * scale + rel[b, a]
            top = max(0.0, float(s.max()))
            e = np.exp(s - top)
            out[i, a] = (e @ v[lo:i + 1, g]) / (math.exp(-top) + e.sum())
    return out


def projections(h, w, prefix, eps):
    """(q, k, v) rows [T, ...]: product and bias, short convolution, then the norms over all of q and all of k."""
    rows = {}
    for n in "qkv":
        u = h @ w[prefix + n].T + w[prefix + n + ".b"]
        rows[n] = short_conv(u, w[prefix + n + ".conv"]) if prefix + n + ".conv" in w else u
    return rms_norm(rows["q"], w[prefix + "q.norm"], eps), rms_norm(rows["k"], w[prefix + "k.norm"], eps), rows["v"]


def attention(h, w, prefix, m, eps, shared):
    """shared: what the first layer with `v_mix` leaves for the later ones (its values)."""
    T = h.shape[0]
    H, G, d = m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    vd = m.get("vdim", d)
    q, k, v = projections(h, w, prefix, eps)
    if m.get("v_mix"):
        if "v" in shared:
            lam = float(w[prefix + "vmix"])
            v = (1.0 - lam) * v + lam * shared["v"]
        else:
            shared["v"] = v
    size = m["mask"]["size"] if m.get("mask") else None
    o = attend(q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, vd), m["scale"], w[prefix + "rel"], m["bias_max"], size)
    return o.reshape(T, H * vd) @ w[prefix + "o"].T


def limited(h, w, prefix, limit):
    g = np.minimum(h @ w[prefix + "gate"].T, limit)
    u = np.clip(h @ w[prefix + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[prefix + "down"].T


def expert(h, w, prefix):
    g = h @ w[prefix + "gate"].T
    return (g * sigmoid(g) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def router(h, w, prefix, r):
    """Chosen experts [T, top], their weights, and each token's margin: the smaller of the gap between the last group kept and
    the first not kept and the gap between the last expert chosen and the first not chosen among the kept groups'."""
    s = sigmoid(h @ w[prefix + "router"].T)
    T, E = s.shape
    top, groups = r["top"], r.get("groups")
    chosen, weight, margin = np.zeros((T, top), dtype=int), np.zeros((T, top)), np.full(T, np.inf)
    for t in range(T):
        allowed = list(range(E))
        if groups:
            size = E // groups["count"]
            score = [sum(sorted(s[t, g * size:(g + 1) * size])[-2:]) for g in range(groups["count"])]
            order = sorted(range(groups["count"]), key=lambda g: -score[g])
            kept = order[:groups["keep"]]
            if groups["keep"] < groups["count"]:
                margin[t] = score[order[groups["keep"] - 1]] - score[order[groups["keep"]]]
            allowed = [e for e in range(E) if e // size in kept]
        order = sorted(allowed, key=lambda e: -s[t, e])
        if top < len(order):
            margin[t] = min(margin[t], s[t, order[top - 1]] - s[t, order[top]])
        chosen[t] = order[:top]
        weight[t] = s[t, chosen[t]] / (s[t, chosen[t]].sum() + 1e-20)
    return chosen, weight, margin


def feed_forward(h, w, prefix, f, margins=None):
    if f["kind"] == "dense":
        return limited(h, w, prefix, f["limit"])
    chosen, weight, margin = router(h, w, prefix, f["router"])
    if margins is not None:
        margins.append(margin)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for k, e in enumerate(chosen[t]):
            out[t] += weight[t, k] * expert(h[t], w, prefix + f"e{int(e)}.")
    if f.get("shared"):
        out += expert(h, w, prefix + "shared.") * sigmoid(h @ w[prefix + "shared.sg"].reshape(-1))[:, None]
    return out


def read_copies(x, w, prefix):
    return np.einsum("s,sti->ti", w[prefix + "in"], x)


def write_copies(x, y, w, prefix):
    return np.einsum("st,sai->tai", w[prefix + "mix"], x) + w[prefix + "out"][:, None, None] * y[None]


def forward(cfg, w, ids, margins=None, streams=None):
    """float64 logits [T, vocab]; margins: list that receives every routed layer's per-token margin;
    streams: list that receives the sum of the copies after every layer."""
    ids = np.asarray(ids)
    x = np.stack([w["embed"][ids] + w["pos"][:len(ids)]] * cfg["streams"])        # [S, T, width]
    eps, shared = cfg["norm"]["eps"], {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = attention(rms_norm(read_copies(x, w, p + "hc1."), w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps, shared)
        x = write_copies(x, y, w, p + "hc1.")
        if layer.get("mlp") is not None:
            y = feed_forward(rms_norm(read_copies(x, w, p + "hc2."), w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], margins)
            x = write_copies(x, y, w, p + "hc2.")
        if streams is not None:
            streams.append(x.sum(axis=0))
    return rms_norm(x.sum(axis=0), w["final.norm"], eps) @ w["head"].T


def min_margin(cfg, w, ids):
    margins = []
    forward(cfg, w, ids, margins)
    return min((float(m.min()) for m in margins), default=math.inf)
