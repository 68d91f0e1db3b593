"""Plain restatement of the Lepalorn decoder for the parity tests: one function per mechanism, whole sequences at once,
no cache, numpy in float64 unless told otherwise. It shares no code with the product.

Weights are a dict name -> array (bfloat16 values widened to float), configuration is the dict of config.json. The
residual stream of every layer comes back beside the logits, so that a test can find the first layer that differs.
"""
from __future__ import annotations

import numpy as np


def rms_normalise(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_rms_norm(x, gain, eps):
    """RMS norm whose gain is one number for all coordinates."""
    return rms_normalise(x, eps) * np.asarray(gain).reshape(())


def vector_rms_norm(x, weight, eps):
    return rms_normalise(x, eps) * weight


def rotate_interleaved(x, positions, base):
    """x[..., T, R]: coordinates 2i and 2i + 1 turned by the angle position * base^(-2i / R)."""
    R = x.shape[-1]
    inv = np.asarray(base, np.float64) ** (-np.arange(0, R, 2, dtype=np.float64) / R)
    ang = positions.astype(np.float64)[:, None] * inv[None, :]
    c, s = np.cos(ang).astype(x.dtype), np.sin(ang).astype(x.dtype)
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def window_mask(T, size):
    """True where query i sees key j: j in [i - size + 1, i]."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < size)


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def latent_of(h, W, p, mix, eps, positions):
    """The two things a latent cache keeps per token: the normed latent and the rotated key part shared by the heads."""
    kv = h @ W[p + "dkv"].T
    r = mix["kv_rank"]
    c = vector_rms_norm(kv[:, :r], W[p + "dkv.norm"], eps)
    return c, rotate_interleaved(kv[:, r:], positions, mix["rot"]["base"])


def latent_attention(h, W, p, mix, latent, positions):
    """h [T, width], latent = (c [T, rank], kr [T, rot]) of this layer or of the one it borrows from."""
    H, D, R, V = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    T = h.shape[0]
    c, kr = latent
    q = (h @ W[p + "q"].T).reshape(T, H, D + R).transpose(1, 0, 2)
    q_rot = rotate_interleaved(q[..., D:], positions, mix["rot"]["base"])
    k = (c @ W[p + "uk"].T).reshape(T, H, D).transpose(1, 0, 2)
    v = (c @ W[p + "uv"].T).reshape(T, H, V).transpose(1, 0, 2)
    s = (q[..., :D] @ k.transpose(0, 2, 1) + q_rot @ kr.T) * mix["scale"]
    s = np.where(window_mask(T, mix["mask"]["size"])[None], s, -np.inf)
    o = softmax(s) @ v                                            # [H, T, V]
    o = o * sigmoid(h @ W[p + "g"].T).T[:, :, None]
    return o.transpose(1, 0, 2).reshape(T, H * V) @ W[p + "o"].T


def clamped_expert(h, W, p, limit):
    g = np.minimum(h @ W[p + "gate"].T, limit)
    u = np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def route(h, W, p, top):
    """Chosen experts [T, top] and their weights: the softmax over the chosen logits."""
    z = h @ W[p + "router"].T + W[p + "router.b"]
    pick = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return pick, softmax(np.take_along_axis(z, pick, axis=-1))


def mixture(h, W, p, mlp):
    pick, w = route(h, W, p, mlp["router"]["top"])
    y = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, col = np.nonzero(pick == e)
        if rows.size:
            y[rows] += w[rows, col][:, None] * clamped_expert(h[rows], W, f"{p}e{e}.", mlp["expert"]["limit"])
    if mlp.get("shared"):
        y += sigmoid(h @ W[p + "shared.sg"].T) * clamped_expert(h, W, p + "shared.", mlp["shared"]["limit"])
    return y


def depth_average(history, coef):
    return sum(a * X for a, X in zip(np.asarray(coef), history))


def forward(cfg, W, ids, dtype=np.float64):
    """Logits [T, vocab] of one sequence and the stream after every layer [layers, T, width]."""
    W = {k: np.asarray(v, dtype) for k, v in W.items()}
    ids = np.asarray(ids, np.int64)
    pos = np.arange(len(ids))
    eps = cfg["norm"]["eps"]
    x = (W["embed"][ids] * dtype(cfg["embedding"]["scale"])).astype(dtype)
    history, latents, stream = [x], {}, []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = layer["mixer"]
        src = mix.get("kv_from")
        if src is None:
            src = i
            latents[i] = latent_of(x, W, p + "mix.", mix, eps, pos)
        x = x + scalar_rms_norm(latent_attention(x, W, p + "mix.", mix, latents[src], pos), W[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + scalar_rms_norm(mixture(x, W, p + "mlp.", layer["mlp"]), W[p + "norm2"], eps)
        history.append(x)
        x = depth_average(history, W[p + "dwa"])
        stream.append(x)
    return scalar_rms_norm(x, W["final.norm"], eps) @ W["head"].T, np.stack(stream)
