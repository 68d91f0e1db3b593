"""Small Tedelix configurations and weights for the tests, made here (not by the package's synthetic builder), so that every
size differs from every other where the design allows it. Weights are bf16-representable float32 arrays."""
import numpy as np

from plan_models import bf16, error, tokens  # noqa: F401  (the tests take them from here)


def attention(heads=6, kv_heads=2, dim=20, vdim=12, rot=8, window=13, scale=None, base=300.0, ff=52):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5, "mask": {"size": window},
         "rot": {"base": base, "dims": rot}}
    return layer("attention", m, ff)


def lightning(heads=3, dim=24, vdim=20, decay=None, ff=44):
    d = decay if decay is not None else [float(x) for x in np.linspace(0.5, 0.99, heads)]
    return layer("lightning", {"heads": heads, "dim": dim, "vdim": vdim, "decay": d}, ff)


def delta(heads=3, dim=20, rank=6, ff=36):
    """rank is no entry of the configuration: the tensors' shapes tell it."""
    out = layer("general_delta", {"heads": heads, "dim": dim}, ff)
    out["mixer"]["_rank"] = rank
    return out


def layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, vocab=151, width=88, eps=1e-5, scale=0.6, softcap=25.0):
    return {"architecture": "Tedelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale, "logit_softcap": softcap,
            "layers": layers}


def varied():
    """Every layer different: groups of one to nine query heads, windows from one key to more than any test's context, partial
    and full rotation, decays from none to forgetting at once, one head, low ranks from one up, no feed-forward."""
    return config([
        delta(heads=2, dim=36, rank=9, ff=70),
        attention(heads=6, kv_heads=2, dim=20, vdim=28, rot=12, window=29, base=90.0, ff=None),
        lightning(heads=5, dim=12, vdim=40, decay=[0.0, 0.3, 0.9, 0.995, 1.0], ff=33),
        attention(heads=9, kv_heads=1, dim=16, vdim=6, rot=16, window=5, ff=20),
        delta(heads=1, dim=50, rank=1, ff=None),
        attention(heads=2, kv_heads=2, dim=44, vdim=18, rot=0, window=4000, ff=61),
        lightning(heads=9, dim=7, vdim=5, ff=None),
        delta(heads=5, dim=9, rank=70, ff=8),
        attention(heads=1, kv_heads=1, dim=6, vdim=34, rot=2, window=1, ff=12),
    ], vocab=153, width=90)


def weights(cfg, seed=0, sharp=1.0, loud=1.0):
    """Random weights; `sharp` scales the queries, so that attention concentrates on few keys; `loud` what the sublayers add to
    the stream: with the table as output head a quiet model repeats its last token."""
    r = np.random.default_rng(seed)
    W = {}

    def mat(name, n, k, gain=1.0):
        W[name] = bf16(r.standard_normal((n, k)) * gain / np.sqrt(k))

    def vec(name, v):
        W[name] = bf16(np.asarray(v, np.float32))

    w = cfg["width"]
    mat("embed", cfg["vocab"], w, 1.5 * np.sqrt(w))
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        H, D = m["heads"], m["dim"]
        vec(f"l{i}.norm1", 1 + 0.3 * r.standard_normal(w))
        if l["type"] == "attention":
            G, V = m["kv_heads"], m["vdim"]
            mat(p + "q", H * D, w, sharp)
            mat(p + "k", G * D, w)
            mat(p + "v", G * V, w)
        else:
            V = m.get("vdim", D)
            mat(p + ("q" if l["type"] == "lightning" else "r"), H * D, w)
            mat(p + "k", H * D, w)
            mat(p + "v", H * V, w)
            mat(p + "g", H * V, w)
            vec(p + "norm", 1 + 0.3 * r.standard_normal(H * V))
            if l["type"] == "general_delta":
                mat(p + "a", H * D, w)
                vec(p + "a.b", 0.7 * r.standard_normal(H * D))
                mat(p + "w1", m["_rank"], w, 1.5)
                mat(p + "w2", H * D, m["_rank"], 1.5)
                vec(p + "w0", -2 + 2 * r.standard_normal(H * D))
        mat(p + "o", w, H * V, 2.0 * loud)
        if l["mlp"]:
            mat(f"l{i}.mlp.up", l["mlp"]["ff"], w)
            mat(f"l{i}.mlp.down", w, l["mlp"]["ff"], loud)
    vec("final.norm", 1 + 0.3 * r.standard_normal(w))
    return W


def alone(l, W, keep):
    """A one-layer model's weights with the other sublayer's output projection at zero."""
    W = dict(W)
    for n in {"mixer": ["l0.mlp.down"], "ff": ["l0.mix.o"], "neither": ["l0.mlp.down", "l0.mix.o"]}[keep]:
        if n in W:
            W[n] = np.zeros_like(W[n])
    return W


# ── one token that stands out ───────────────────────────────────────────────
MARK, PLAIN = 0, 1


def _marker_embedding(W):
    e = W["embed"]
    e[:, 0], e[:, 1] = 0.0, 4.0
    e[MARK, 0] = 60.0
    for n in W:
        if n.endswith("norm1"):
            W[n][:2] = 1.0


def marker_attention(window, heads=6, kv_heads=2):
    """Every query looks for the marker token along a coordinate that is not rotated: a visible marker takes all of the
    attention, an invisible one leaves a broad mixture."""
    cfg = config([attention(heads=heads, kv_heads=kv_heads, dim=18, vdim=14, rot=8, window=window, scale=0.25, ff=None)], width=64)
    W = weights(cfg, seed=21)
    _marker_embedding(W)
    q, k = W["l0.mix.q"].reshape(heads, 18, -1), W["l0.mix.k"].reshape(kv_heads, 18, -1)
    q[:, 17], k[:, 17] = 0.0, 0.0
    q[:, 17, 1], k[:, 17, 0] = 12.0, 1.0
    return cfg, {n: bf16(v) for n, v in W.items()}


def marker_state(kind, heads=3):
    """Only the marker writes into the states, which keep it for good: without it every later output is another one."""
    cfg = config([lightning(heads=heads, dim=12, vdim=18, decay=[1.0] * heads, ff=None) if kind == "lightning" else delta(heads=heads, dim=18, rank=3, ff=None)],
                 width=64)
    W = weights(cfg, seed=22)
    _marker_embedding(W)
    D = cfg["layers"][0]["mixer"]["dim"]
    k, q = W["l0.mix.k"].reshape(heads, D, -1), W["l0.mix." + ("q" if kind == "lightning" else "r")].reshape(heads, D, -1)
    k[:], k[:, 1, 0] = 0.0, 1.0
    q[:, 1], q[:, 1, 1] = 0.0, 4.0
    if kind == "general_delta":
        W["l0.mix.w0"][:] = -30.0
    return cfg, {n: bf16(v) for n, v in W.items()}
