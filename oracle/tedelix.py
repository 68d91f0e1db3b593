"""Plain restatement of the Tedelix decoder for the parity tests: one function per mechanism, whole sequences at once, no
cache and no chunks (recurrences go token by token), numpy in float64 unless told otherwise. It shares no code with the
product.

Weights are a dict name -> array (bfloat16 values widened to float), configuration is the dict of config.json. The residual
stream after every layer comes back beside the logits, so that a test can find the first layer that differs.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


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


# ── attention ───────────────────────────────────────────────────────────────
def angles(positions, dims, base):
    """[T, dims / 2]: position * base^(-2 i / dims)."""
    inv = np.asarray(base, np.float64) ** (-np.arange(0, dims, 2, dtype=np.float64) / dims)
    return positions.astype(np.float64)[:, None] * inv[None, :]


def rotate_halves(x, positions, dims, base):
    """x[..., T, D]: coordinates i and i + dims / 2 of the first `dims` are turned together; the rest pass."""
    a = angles(positions, dims, base)
    c, s = np.cos(a).astype(x.dtype), np.sin(a).astype(x.dtype)
    u, v = x[..., : dims // 2], x[..., dims // 2: dims]
    out = np.array(x)
    out[..., : dims // 2] = u * c - v * s
    out[..., dims // 2: dims] = v * c + u * s
    return out


def window_mask(T, size):
    """True where query i sees key j: i - size < j <= i."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < size)


def rotated_values(v, positions, base):
    return rotate_halves(v, positions, v.shape[-1], base)


def turned_back(o, positions, base):
    return rotate_halves(o, -positions, o.shape[-1], base)


def attention(h, W, p, mix, eps, positions):
    """The mixture of values before the output projection, [T, heads * vdim]."""
    T, H, G, D, V = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    base, dims = mix["rot"]["base"], mix["rot"]["dims"]
    heads = lambda name, n, d: (h @ W[p + name].T).reshape(T, n, d).transpose(1, 0, 2)  # noqa: E731
    q = rotate_halves(heads("q", H, D), positions, dims, base)
    k = rotate_halves(heads("k", G, D), positions, dims, base)
    v = rotated_values(heads("v", G, V), positions, base)
    k, v = np.repeat(k, H // G, axis=0), np.repeat(v, H // G, axis=0)
    s = np.where(window_mask(T, mix["mask"]["size"])[None], (q @ k.transpose(0, 2, 1)) * mix["scale"], -np.inf)
    o = turned_back(softmax(s) @ v, positions, base)
    return o.transpose(1, 0, 2).reshape(T, H * V)


# ── recurrences ─────────────────────────────────────────────────────────────
def lightning_scan(q, k, v, decay):
    """q, k [H, T, D], v [H, T, V]: S <- decay S + k v^T, o = S^T q."""
    S = np.zeros((q.shape[0], q.shape[2], v.shape[2]), q.dtype)
    o = np.empty_like(v)
    for t in range(q.shape[1]):
        S = decay[:, None, None] * S + k[:, t, :, None] * v[:, t, None, :]
        o[:, t] = np.einsum("hdv,hd->hv", S, q[:, t])
    return o


def lightning(h, W, p, mix, eps, positions):
    T, H, D, V = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    part = lambda name, d: silu(h @ W[p + name].T).reshape(T, H, d).transpose(1, 0, 2)  # noqa: E731
    o = lightning_scan(part("q", D), part("k", D), part("v", V), np.asarray(mix["decay"], h.dtype))
    o = rms(o.transpose(1, 0, 2).reshape(T, H * V), eps) * W[p + "norm"]
    return o * sigmoid(h @ W[p + "g"].T)


def channel_decay(h, W, p):
    """exp(-e^(-1/2) sigmoid(low-rank logit)), in (0.545, 1)."""
    z = np.tanh(h @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"]
    return np.exp(-np.exp(-0.5) * sigmoid(z))


def removal_rate(h, W, p):
    return sigmoid(h @ W[p + "a"].T + W[p + "a.b"])


def unit_key(k):
    return k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + 1e-6)


def delta_scan(r, k, v, w, a):
    """All [H, T, D]: S <- diag(w) S - (a u)(u^T S) + k v^T with the unit key u, o = S^T r."""
    u = unit_key(k)
    S = np.zeros((r.shape[0], r.shape[2], v.shape[2]), r.dtype)
    o = np.empty_like(v)
    for t in range(r.shape[1]):
        held = np.einsum("hd,hdv->hv", u[:, t], S)
        S = w[:, t, :, None] * S - (a[:, t] * u[:, t])[:, :, None] * held[:, None, :] + k[:, t, :, None] * v[:, t, None, :]
        o[:, t] = np.einsum("hdv,hd->hv", S, r[:, t])
    return o


def general_delta(h, W, p, mix, eps, positions):
    T, H, D = h.shape[0], mix["heads"], mix["dim"]
    heads = lambda y: y.reshape(T, H, D).transpose(1, 0, 2)  # noqa: E731
    r, k, v = (heads(h @ W[p + n].T) for n in ("r", "k", "v"))
    o = delta_scan(r, k, v, heads(channel_decay(h, W, p)), heads(removal_rate(h, W, p)))
    o = rms(o, eps).transpose(1, 0, 2).reshape(T, H * D) * W[p + "norm"]
    return o * sigmoid(h @ W[p + "g"].T)


# ── the model ───────────────────────────────────────────────────────────────
MIXERS = {"attention": attention, "lightning": lightning, "general_delta": general_delta}


def feed_forward(h, W, p):
    return squared_relu(h @ W[p + "up"].T) @ W[p + "down"].T


def output_logits(x, W, cfg):
    z = (rms(x, cfg["norm"]["eps"]) * W["final.norm"]) @ W["embed"].T * cfg["logit_scale"]
    return cfg["logit_softcap"] * np.tanh(z / cfg["logit_softcap"])


def forward(cfg, W, ids, dtype=np.float64):
    """Logits [T, vocab] of one sequence and the stream after every layer [layers, T, width]."""
    W = {k: np.asarray(v, dtype) for k, v in W.items()}
    ids = np.asarray(ids, np.int64)
    pos, eps = np.arange(len(ids)), cfg["norm"]["eps"]
    x, stream = W["embed"][ids], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * W[p + "norm1"]
        y = MIXERS[layer["type"]](h, W, p + "mix.", layer["mixer"], eps, pos) @ W[p + "mix.o"].T
        if layer.get("mlp"):
            y = y + feed_forward(h, W, p + "mlp.")
        x = x + y
        stream.append(x)
    return output_logits(x, W, cfg), np.stack(stream)
