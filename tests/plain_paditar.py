"""Plain, slow Paditar in numpy: the oracle the engine is compared with.

Whole sequences, no cache, no batching, float64, one function per mechanism, token by token where that is how the mechanism is
defined, written from the design's equations; it shares no code with the package (only the file readers of the other oracle).

    x = E[token];  layers 0 .. start - 1;
    for t = 0 .. times - 1:  (t > 0: x <- x + E[token]);  x <- x + step[t];  layers start .. stop - 1 (the same weights every time)
    layers stop .. ;  logits = E n(x; final)
    layer:  x <- x + n(mixer(n(x)));  x <- x + n(W_down max(W_up n(x), 0)^2)        n(v; w) = v / sqrt(mean(v^2) + eps) (1 + w)
"""
from __future__ import annotations

import math
import os

import numpy as np

from plain_gemma2 import read_config, read_safetensors  # noqa: F401  (file formats only)


def load_folder(folder):
    w = read_safetensors(os.path.join(folder, "model.safetensors"))
    return read_config(folder), {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}


def exact(x):
    return x


def noise(size, seed):
    """A stand-in for rounding: every value moved by up to `size` of itself.  Passed to `forward`, it shows how far rounding alone
    moves the logits at each position: designs that divide small differences by their own root mean square amplify it unevenly."""
    rng = np.random.default_rng(seed)
    return lambda x: x * (1.0 + size * rng.uniform(-1.0, 1.0, size=x.shape))


def to_bfloat16(x):
    """Every value rounded to bfloat16 (to nearest, ties to even)."""
    bits = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & np.uint32(0xFFFF0000)
    return bits.view(np.float32).astype(np.float64)


def unit(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    """The weight holds the scale minus one."""
    return unit(x, eps) * (1.0 + w)


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


def rotate(x, base, n):
    """x [T, ..., d]: pairs (i, i + n/2) of the first n values turned by position * base^(-2 i / n)."""
    out = x.copy()
    for p in range(x.shape[0]):
        for i in range(n // 2):
            a = p * base ** (-2.0 * i / n)
            u, v = x[p, ..., i], x[p, ..., i + n // 2]
            out[p, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[p, ..., i + n // 2] = v * math.cos(a) + u * math.sin(a)
    return out


def temperature(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def attend(q, k, v, scale, extra):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]: causal softmax of scale * (q . k) with `extra` (0 or 1) added to the
    denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for a in range(H):
            g = a // (H // G)
            s = k[:i + 1, g] @ q[i, a] * scale
            top = float(s.max()) if extra == 0 else max(0.0, float(s.max()))
            e = np.exp(s - top)
            out[i, a] = (e @ v[:i + 1, g]) / (extra * math.exp(-top) + e.sum())
    return out


def layer_lambda(w, prefix, diff):
    return math.exp(float(w[prefix + "lq1"] @ w[prefix + "lk1"])) - math.exp(float(w[prefix + "lq2"] @ w[prefix + "lk2"])) + diff


def differential(q, k, v, scale, lam, r=exact):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, e]: the difference of the two maps' outputs."""
    a1 = attend(q[:, :, 0], k[:, :, 0], v, scale, 0)
    a2 = attend(q[:, :, 1], k[:, :, 1], v, scale, 0)
    return r(a1) - lam * r(a2)


def differential_attention(h, w, prefix, m, eps, r=exact):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, e = m.get("kv_heads", H), m.get("vdim", d)
    q = r(rotate(r(h @ w[prefix + "q"].T).reshape(T, H, 2, d), m["rot"]["base"], m["rot"]["dims"]))
    k = r(rotate(r(h @ w[prefix + "k"].T).reshape(T, G, 2, d), m["rot"]["base"], m["rot"]["dims"]))
    v = r(h @ w[prefix + "v"].T).reshape(T, G, e)
    o = differential(q, k, v, m["scale"], layer_lambda(w, prefix, m["diff"]), r)
    o = unit(o, eps) * (1.0 - m["diff"])
    return r(o.reshape(T, H * e) * sigmoid(r(h @ w[prefix + "g"].T))) @ w[prefix + "o"].T


def key_value_attention(h, w, prefix, m, eps, r=exact):
    """Attention whose values are its keys as the convolution leaves them."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G = m.get("kv_heads", H)
    q = short_conv(r(h @ w[prefix + "q"].T) + w[prefix + "q.b"], w[prefix + "q.conv"]).reshape(T, H, d)
    k = short_conv(r(h @ w[prefix + "k"].T) + w[prefix + "k.b"], w[prefix + "k.conv"]).reshape(T, G, d)
    v = r(k)
    q, k = unit(q, eps) * w[prefix + "q.norm"], r(unit(k, eps) * w[prefix + "k.norm"])
    q = q * np.array([temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"]) for p in range(T)])[:, None, None]
    o = attend(r(q), k, v, m["scale"], 1)
    o = r(r(o) * sigmoid(r(h @ w[prefix + "g"].T))[:, :, None])
    return o.reshape(T, H * d) @ w[prefix + "o"].T + w[prefix + "o.b"]


def memory(q, k, v, zi, zf, cap, den_eps=1e-6, state=None):
    """The recurrence of one head: q, k [T, d] (q scaled), v [T, e], gate logits zi, zf [T] -> o [T, e]; state: (S, n, m) to start
    from (zeros), returned as well."""
    S, n, m = state if state is not None else (np.zeros((k.shape[1], v.shape[1])), np.zeros(k.shape[1]), 0.0)
    out = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        i = cap * math.tanh(zi[t] / cap)
        f = -math.log1p(math.exp(-cap * math.tanh(zf[t] / cap)))
        new = max(f + m, i)
        S = math.exp(f + m - new) * S + math.exp(i - new) * np.outer(k[t], v[t])
        n = math.exp(f + m - new) * n + math.exp(i - new) * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + den_eps)
    return out, (S, n, m)


def memory_mixer(h, w, prefix, m, eps, r=exact):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    e = m.get("vdim", d)
    q = r(h @ w[prefix + "q"].T).reshape(T, H, d) * d ** -0.5
    k = r(h @ w[prefix + "k"].T).reshape(T, H, d)
    v = r(h @ w[prefix + "v"].T).reshape(T, H, e)
    zi, zf = r(h @ w[prefix + "i"].T) + w[prefix + "i.b"], r(h @ w[prefix + "f"].T) + w[prefix + "f.b"]
    o = np.stack([memory(q[:, a], k[:, a], v[:, a], zi[:, a], zf[:, a], m["gate_cap"])[0] for a in range(H)], axis=1)
    o = unit(r(o), eps).reshape(T, H * e) * w[prefix + "norm"] * sigmoid(r(h @ w[prefix + "g"].T))
    return r(o) @ w[prefix + "o"].T


def mixer(h, w, prefix, layer, eps, r=exact):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return differential_attention(h, w, prefix, m, eps, r)
    return m["left_scale"] * key_value_attention(h, w, prefix + "left.", m["left"], eps, r) + \
        m["right_scale"] * memory_mixer(h, w, prefix + "right.", m["right"], eps, r)


def feed_forward(h, w, prefix, r=exact):
    u = np.maximum(h @ w[prefix + "up"].T, 0.0)
    return r(u * u) @ w[prefix + "down"].T


def run_layer(x, w, i, layer, eps, r=exact):
    p = f"l{i}."
    x = x + rms_norm(r(mixer(r(rms_norm(x, w[p + "norm1"], eps)), w, p + "mix.", layer, eps, r)), w[p + "norm1b"], eps)
    if layer.get("mlp") is not None:
        x = x + rms_norm(r(feed_forward(r(rms_norm(x, w[p + "norm2"], eps)), w, p + "mlp.", r)), w[p + "norm2b"], eps)
    return x


def forward(cfg, w, ids, streams=None, r=exact):
    """float64 logits [T, vocab]; streams: list that receives the stream after every layer run; r: what stands in for rounding
    where a 16-bit implementation would round."""
    x = embedded = w["embed"][np.asarray(ids)]
    eps, layers, loop = cfg["norm"]["eps"], cfg["layers"], cfg.get("loop")

    def run(x, first, last):
        for i in range(first, last):
            x = run_layer(x, w, i, layers[i], eps, r)
            if streams is not None:
                streams.append(x)
        return x
    if loop is None:
        x = run(x, 0, len(layers))
    else:
        x = run(x, 0, loop["start"])
        for t in range(loop["times"]):
            if t > 0:
                x = x + embedded
            x = run(x + w["loop.step"][t], loop["start"], loop["stop"])
        x = run(x, loop["stop"], len(layers))
    return r(rms_norm(x, w["final.norm"], eps)) @ w["embed"].T
