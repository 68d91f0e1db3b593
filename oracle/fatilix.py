"""Plain restatement of the Fatilix decoder for the parity tests: one function per mechanism, whole sequences at once, no
cache, numpy in float64 unless told otherwise. It shares no code with the product.

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


def squared_relu(z):
    return np.square(np.maximum(z, 0.0))


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose weight is kept as its distance from one."""
    return rms(x, eps) * (1.0 + w)


# ── what enters ─────────────────────────────────────────────────────────────
def embedding(ids, W, scale):
    return W["embed"][ids] * scale + W["pos"][: len(ids)]


# ── attention ───────────────────────────────────────────────────────────────
def temperature(positions, coef, every):
    """Factor of the queries: grows by steps, one every `every` positions."""
    return 1.0 + coef * np.log(np.floor((positions + 1.0) / every) + 1.0)


def bucket(distance, rows, far):
    """Row of the bias table: one per distance up to half of the rows, then logarithmic up to distance `far`."""
    half = rows // 2
    if distance < half:
        return distance
    return min(rows - 1, half + int(math.floor(math.log(distance / half) / math.log(far / half) * (rows - half))))


def distance_bias(table, far, T):
    """[heads, T, T]: table[bucket(i - j)] per head where j <= i."""
    by_distance = np.stack([table[bucket(n, len(table), far)] for n in range(T)])
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return by_distance[np.maximum(d, 0)].transpose(2, 0, 1)


def causal(T):
    return np.arange(T)[:, None] >= np.arange(T)[None, :]


def sink_weights(scores, sink):
    """Softmax of [H, T, T] scores along the last axis whose denominator has one term more per head."""
    m = np.maximum(scores.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(scores - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - m))


def split_heads(y, n):
    return y.reshape(y.shape[0], n, -1).transpose(1, 0, 2)


def mix(q, k, v, scores_extra, W, p, m):
    """q [H, T, D], k and v [G, T, .]: the heads' mixtures side by side, [T, H * V]."""
    H, G = m["heads"], m["kv_heads"]
    k, v = np.repeat(k, H // G, axis=0), np.repeat(v, H // G, axis=0)
    s = (q @ k.transpose(0, 2, 1)) * m["scale"] + scores_extra
    s = np.where(causal(q.shape[1])[None], s, -np.inf)
    o = sink_weights(s, W[p + "sink"]) @ v
    return o.transpose(1, 0, 2).reshape(q.shape[1], -1)


def output_gate(o, h, W, p):
    return o * sigmoid(h @ W[p + "g"].T)


def attention(h, W, p, m, eps, positions):
    """Keys serve as values, taken before their norm."""
    k = split_heads(h @ W[p + "k"].T, m["kv_heads"])
    q = rms(split_heads(h @ W[p + "q"].T, m["heads"]), eps) * W[p + "q.norm"]
    q = q * temperature(positions, m["q_temp"]["coef"], m["q_temp"]["every"])[None, :, None]
    o = mix(q, rms(k, eps) * W[p + "k.norm"], k, 0.0, W, p, m)
    return output_gate(o, h, W, p) @ W[p + "o"].T


def attention_2(h, W, p, m, eps, positions):
    """Biased projections, unweighted norms, a learned bias by distance."""
    part = lambda n, heads: split_heads(h @ W[p + n].T + W[p + n + ".b"], heads)  # noqa: E731
    q = rms(part("q", m["heads"]), eps) * temperature(positions, m["q_temp"]["coef"], m["q_temp"]["every"])[None, :, None]
    k, v = rms(part("k", m["kv_heads"]), eps), part("v", m["kv_heads"])
    o = mix(q, k, v, distance_bias(W[p + "rel"], m["bias_max"], len(h)), W, p, m)
    return output_gate(o, h, W, p) @ W[p + "o"].T


# ── feed-forward ────────────────────────────────────────────────────────────
def dense(h, W, p):
    return squared_relu(h @ W[p + "up"].T) @ W[p + "down"].T


def gated_expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def best(values, n):
    """Indices of the n largest along the last axis, the lower index first among equals."""
    return np.argsort(-values, axis=-1, kind="stable")[:, :n]


def allowed_experts(choice, groups, keep):
    """True for the experts of each token's best groups; a group counts by its best expert."""
    T, E = choice.shape
    top = best(choice.reshape(T, groups, E // groups).max(-1), keep)
    ok = np.zeros((T, groups), bool)
    np.put_along_axis(ok, top, True, axis=-1)
    return np.repeat(ok, E // groups, axis=1)


def route(h, W, p, r):
    """Chosen experts and their weights, [T, top] each."""
    s = softmax(h @ W[p + "router"].T)
    choice = s + W[p + "correction"]
    pick = best(np.where(allowed_experts(choice, r["groups"]["count"], r["groups"]["keep"]), choice, -np.inf), r["top"])
    w = np.take_along_axis(s, pick, axis=-1)
    return pick, w / (w.sum(-1, keepdims=True) + 1e-20) * r["scale"]


def experts(h, W, p, mlp):
    pick, w = route(h, W, p, mlp["router"])
    y = gated_expert(h, W, p + "shared.") if mlp.get("shared") else np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, col = np.nonzero(pick == e)
        if rows.size:
            y[rows] += w[rows, col][:, None] * gated_expert(h[rows], W, f"{p}e{e}.")
    return y


# ── the model ───────────────────────────────────────────────────────────────
MIXERS = {"attention": attention, "attention_2": attention_2}


def residual(x, y, w, eps, mult):
    return x + mult * offset_norm(y, w, eps)


def forward(cfg, W, ids, dtype=np.float64):
    """Logits [T, vocab] of one sequence and the stream after every layer [layers, T, width]."""
    W = {k: np.asarray(v, dtype) for k, v in W.items()}
    ids = np.asarray(ids, np.int64)
    pos, eps, mult = np.arange(len(ids)), cfg["norm"]["eps"], cfg["residual_mult"]
    x, stream = embedding(ids, W, cfg["embedding"]["scale"]), []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        # looked up by name, so that a test can replace one mechanism
        mixer = globals()[MIXERS[layer["type"]].__name__]
        x = residual(x, mixer(x, W, p + "mix.", layer["mixer"], eps, pos), W[p + "norm1"], eps, mult)
        mlp = layer.get("mlp")
        if mlp:
            y = dense(x, W, p + "mlp.") if mlp["kind"] == "dense" else experts(x, W, p + "mlp.", mlp)
            x = residual(x, y, W[p + "norm2"], eps, mult)
        stream.append(x)
    return offset_norm(x, W["final.norm"], eps) @ W["head"].T, np.stack(stream)
