"""Plain restatement of the Revelix decoder for the parity tests: one function per mechanism, whole sequences at once, no
cache and no chunks (recurrences go token by token), numpy in float64 unless told otherwise. It shares no code with the
product.

Weights are a dict name -> array (bfloat16 values widened to float), configuration is the dict of config.json. The residual
stream after every layer comes back beside the logits, so that a test can find the first layer that differs.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def xielu(z, p, q):
    """z / 2 plus a parabola on the right, an exponential less its tangent on the left."""
    return z / 2 + np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(np.minimum(z, 0.0)) - np.minimum(z, 0.0)))


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def tanh_norm(x, W, name):
    """The stream's norm: no statistics, a tanh with a learned slope."""
    return np.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def split_heads(y, n):
    """[T, n * d] -> [n, T, d]"""
    return y.reshape(y.shape[0], n, -1).transpose(1, 0, 2)


def join_heads(o):
    return o.transpose(1, 0, 2).reshape(o.shape[1], -1)


# ── rotation ────────────────────────────────────────────────────────────────
def frequencies(dims, base):
    return float(base) ** (-np.arange(0, dims, 2, dtype=np.float64) / dims)


def stretched_frequencies(dims, base, factor, original, fast, slow):
    """Pairs that turn often within the original length keep their frequency, slow ones have it divided by factor, linear between."""
    at = lambda turns: dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(at(fast)), 0), min(math.ceil(at(slow)), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    f = frequencies(dims, base)
    return f / factor * ramp + f * (1 - ramp)


def magnitude(scaling):
    return 0.1 * math.log(scaling["factor"]) + 1.0 if scaling else 1.0


def rotate(x, positions, rot, pairs):
    """x[..., T, D]: the first rot.dims coordinates in pairs, neighbours (pairs) or i and i + dims / 2; the rest pass."""
    n, scaling = rot["dims"], rot.get("scaling")
    f = stretched_frequencies(n, rot["base"], **scaling) if scaling else frequencies(n, rot["base"])
    a = positions.astype(np.float64)[:, None] * f[None, :]
    c, s = (np.cos(a) * magnitude(scaling)).astype(x.dtype), (np.sin(a) * magnitude(scaling)).astype(x.dtype)
    first, second = (slice(0, n, 2), slice(1, n, 2)) if pairs else (slice(0, n // 2), slice(n // 2, n))
    out = np.array(x)
    out[..., first] = x[..., first] * c - x[..., second] * s
    out[..., second] = x[..., second] * c + x[..., first] * s
    return out


# ── retention ───────────────────────────────────────────────────────────────
def decaying_sum(q, k, v, decay):
    """q, k [H, T, D], v [H, T, V]: S <- decay S + k v^T, o = S^T q."""
    S = np.zeros((q.shape[0], q.shape[2], v.shape[2]), q.dtype)
    o = np.empty_like(v)
    for t in range(q.shape[1]):
        S = decay[:, None, None] * S + k[:, t, :, None] * v[:, t, None, :]
        o[:, t] = np.einsum("hdv,hd->hv", S, q[:, t])
    return o


def retention(h, W, p, mix, eps, positions):
    H, D = mix["heads"], mix["dim"]
    q, k, v = (split_heads(h @ W[p + n].T, H) for n in "qkv")
    q, k = rotate(q, positions, mix["rot"], False), rotate(k, positions, mix["rot"], False) * D ** -0.5
    o = rms(decaying_sum(q, k, v, np.asarray(mix["decay"], h.dtype)), eps)
    return (join_heads(o) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ── the left mixer: attention ───────────────────────────────────────────────
def short_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1]), u.dtype), u])
    return sum(padded[j: j + len(u)] * w[:, j] for j in range(taps))


def kept_window_mask(T, size, keep):
    """True where query i sees key j: the last `size` keys and the sequence's first `keep`."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < size) | (np.arange(T)[None, :] < keep))


def capped(s, cap):
    return cap * np.tanh(s / cap)


def sink_weights(scores, sink):
    """Softmax of [H, T, T] scores along the last axis whose denominator has one term more per head."""
    m = np.maximum(scores.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(scores - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - m))


def mixed_heads(weights, talk):
    """weights [H, T, T]: head h's become sum over g of talk[h, g] weights[g]."""
    return np.einsum("hg,gij->hij", talk, weights)


def attention(h, W, p, mix, eps, positions):
    H, G = mix["heads"], mix["kv_heads"]
    q, k, v = (short_conv(h @ W[p + n].T + W[p + n + ".b"], W[p + n + ".conv"]) for n in "qkv")
    q, k, v = rotate(split_heads(q, H), positions, mix["rot"], True), rotate(split_heads(k, G), positions, mix["rot"], True), split_heads(v, G)
    k, v = np.repeat(k, H // G, axis=0), np.repeat(v, H // G, axis=0)
    s = capped((q @ k.transpose(0, 2, 1)) * mix["scale"], mix["softcap"])
    s = np.where(kept_window_mask(len(h), mix["mask"]["size"], mix["mask"]["keep_first"])[None], s, -np.inf)
    w = mixed_heads(sink_weights(s, W[p + "sink"]), W[p + "talk"])
    return join_heads(w @ v) @ W[p + "o"].T


# ── the right mixer: a gated sum ────────────────────────────────────────────
def gated_sum(q, f, v):
    """q, f [H, T, D], v [H, T, V]: S <- diag(f) S + (1 - f) v^T, o = S^T q."""
    S = np.zeros((q.shape[0], q.shape[2], v.shape[2]), q.dtype)
    o = np.empty_like(v)
    for t in range(q.shape[1]):
        S = f[:, t, :, None] * S + (1 - f[:, t])[:, :, None] * v[:, t, None, :]
        o[:, t] = np.einsum("hdv,hd->hv", S, q[:, t])
    return o


def forget(h, W, p):
    """Between the lower bound and one."""
    low = W[p + "lower"]
    return low + (1 - low) * sigmoid(h @ W[p + "f"].T + W[p + "f.b"])


def gated(h, W, p, mix, eps, positions):
    H = mix["heads"]
    o = gated_sum(split_heads(silu(h @ W[p + "q"].T), H), split_heads(forget(h, W, p), H), split_heads(h @ W[p + "v"].T, H))
    return join_heads(rms(o, eps) * W[p + "norm"]) @ W[p + "o"].T


# ── the model ───────────────────────────────────────────────────────────────
def parallel(h, W, p, mix, eps, positions):
    return (mix["left_scale"] * attention(h, W, p + "left.", mix["left"], eps, positions)
            + mix["right_scale"] * gated(h, W, p + "right.", mix["right"], eps, positions))


MIXERS = {"retention": retention, "parallel": parallel}


def feed_forward(h, W, p):
    return xielu(h @ W[p + "up"].T, *np.ravel(W[p + "act"])) @ W[p + "down"].T


def forward(cfg, W, ids, dtype=np.float64):
    """Logits [T, vocab] of one sequence and the stream after every layer [layers, T, width]."""
    W = {k: np.asarray(v, dtype) for k, v in W.items()}
    ids = np.asarray(ids, np.int64)
    pos, eps = np.arange(len(ids)), cfg["norm"]["eps"]
    x, stream = W["embed"][ids], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](tanh_norm(x, W, p + "norm1"), W, p + "mix.", layer["mixer"], eps, pos)
        if layer.get("mlp"):
            x = x + feed_forward(tanh_norm(x, W, p + "norm2"), W, p + "mlp.")
        stream.append(x)
    return tanh_norm(x, W, "final.norm") @ W["embed"].T * cfg["logit_scale"], np.stack(stream)
