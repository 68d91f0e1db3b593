"""Small Revelix configurations and weights for the tests, made here (not by the package's synthetic builder), so that every size
differs from every other where the design allows it. Weights are bf16-representable float32 arrays."""
import numpy as np

from plan_models import bf16, error, tokens  # noqa: F401  (the tests take them from here)


def retention(heads=3, dim=24, vdim=20, rot=16, base=300.0, decay=None, ff=None):
    d = decay if decay is not None else [float(x) for x in np.linspace(0.6, 0.99, heads)]
    return layer("retention", {"heads": heads, "dim": dim, "vdim": vdim, "decay": d, "rot": {"base": base, "dims": rot}}, ff)


SCALING = {"factor": 3.0, "original": 60, "fast": 8.0, "slow": 0.5}


def left(heads=6, kv_heads=2, dim=20, vdim=28, rot=12, base=90.0, scaling=SCALING, window=29, keep=5, conv=3, softcap=9.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5, "softcap": softcap, "conv": conv,
         "mask": {"size": window, "keep_first": keep}, "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(scaling)
    return m


def right(heads=5, dim=14, vdim=11):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def parallel(a=None, b=None, left_scale=0.7, right_scale=1.2, ff=52):
    return layer("parallel", {"left": a or left(), "right": b or right(), "left_scale": left_scale, "right_scale": right_scale}, ff)


def layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, vocab=151, width=88, eps=1e-4, scale=0.6):
    return {"architecture": "Revelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale, "layers": layers}


def varied():
    """Every layer different: either mixer with and without a feed-forward, one to nine query heads per cached head, windows from
    one key to more than any test's context, none to a page and more of kept keys, one to seven taps, full, partial and no
    rotation, stretched and not, decays from none to forgetting at once."""
    return config([
        parallel(left(heads=6, kv_heads=2, dim=20, vdim=28, window=29, keep=5), right(heads=5, dim=14, vdim=11), ff=70),
        retention(heads=5, dim=12, vdim=40, rot=12, decay=[0.0, 0.3, 0.9, 0.995, 1.0]),
        parallel(left(heads=9, kv_heads=1, dim=16, vdim=6, rot=16, window=5, keep=1, conv=1, softcap=3.0), right(heads=1, dim=50, vdim=9), left_scale=1.3, ff=None),
        parallel(left(heads=2, kv_heads=2, dim=44, vdim=17, rot=0, scaling=None, window=4000, keep=0, conv=2, softcap=60.0), right(heads=9, dim=7, vdim=5),
                 right_scale=0.4, ff=33),
        retention(heads=1, dim=50, vdim=7, rot=0, ff=21),
        parallel(left(heads=1, kv_heads=1, dim=6, vdim=34, rot=2, window=1, keep=20, conv=7), right(heads=2, dim=33, vdim=30), ff=12),
        retention(heads=7, dim=9, vdim=5, rot=4, base=3.0, ff=40),
        parallel(left(heads=20, kv_heads=4, dim=10, vdim=12, rot=10, window=37, keep=17, conv=4, scaling={"factor": 1.5, "original": 1000, "fast": 2.0, "slow": 1.0}),
                 right(heads=3, dim=20, vdim=16), ff=None),
    ], vocab=153, width=90, eps=1e-2)


def mixed_layers():
    """One layer of each kind and another parallel one, sizes that are no multiples of anything."""
    return config([parallel(left(heads=6, kv_heads=3, dim=18, vdim=26, rot=10, window=37, keep=3), right(heads=3, dim=22, vdim=13), ff=45),
                   retention(heads=5, dim=14, vdim=11, rot=6, ff=27),
                   parallel(left(heads=10, kv_heads=2, dim=12, vdim=9, window=21, keep=18, conv=4), right(heads=2, dim=30, vdim=25), left_scale=0.9, ff=None)],
                  vocab=133, width=76)


def weights(cfg, seed=0, sharp=1.0, loud=1.0):
    """Random weights; `sharp` scales the queries, so that attention concentrates on few keys; `loud` what the sublayers add to the
    stream. A state's output is divided by its size, so early outputs hang on the sign of one product of query and key: these
    are made to agree (keys like queries, forget-gated queries mostly positive)."""
    r = np.random.default_rng(seed)
    W = {}
    w = cfg["width"]

    def mat(name, n, k, gain=1.0):
        W[name] = bf16(r.standard_normal((n, k)) * gain / np.sqrt(k))

    def vec(name, v):
        W[name] = bf16(np.asarray(v, np.float32))

    def norm(name):
        vec(name, 1 + 0.3 * r.standard_normal(w))
        vec(name + ".b", 0.3 * r.standard_normal(w))
        vec(name + ".alpha", r.uniform(0.3, 1.2))

    mat("embed", cfg["vocab"], w, 1.5 * np.sqrt(w))
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        norm(p + "norm1")
        if l["type"] == "retention":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * D, w)
            W[p + "mix.k"] = bf16(0.8 * W[p + "mix.q"] + 0.6 * r.standard_normal((H * D, w)) / np.sqrt(w))
            mat(p + "mix.v", H * V, w)
            mat(p + "mix.g", H * V, w)
            mat(p + "mix.o", w, H * V, 2.0 * loud)
        else:
            a, b, pl, pr = m["left"], m["right"], p + "mix.left.", p + "mix.right."
            H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, rows, gain in (("q", H * D, sharp), ("k", G * D, 1.0), ("v", G * V, 1.0)):
                mat(pl + n, rows, w, gain)
                vec(pl + n + ".b", 0.5 * r.standard_normal(rows))
                vec(pl + n + ".conv", r.standard_normal((rows, a["conv"])) * a["conv"] ** -0.5)
            vec(pl + "talk", 0.6 * np.eye(H) + r.standard_normal((H, H)) * H ** -0.5)
            vec(pl + "sink", 1.0 + r.standard_normal(H))
            mat(pl + "o", w, H * V, 2.0 * loud)
            H, D, V = b["heads"], b["dim"], b["vdim"]
            shift = W[p + "norm1.b"] / np.sum(W[p + "norm1.b"] ** 2)
            W[pr + "q"] = bf16(r.standard_normal((H * D, w)) / np.sqrt(w) + 1.5 * shift)
            mat(pr + "f", H * D, w, 2.0)
            vec(pr + "f.b", 1 + 2 * r.standard_normal(H * D))
            low = r.uniform(-0.3, 0.95, H * D)
            vec(pr + "lower", np.maximum(low, 0.0))                # a third is free to forget everything
            mat(pr + "v", H * V, w)
            vec(pr + "norm", 1 + 0.3 * r.standard_normal(V))
            mat(pr + "o", w, H * V, loud)
        if l["mlp"]:
            norm(p + "norm2")
            mat(p + "mlp.up", l["mlp"]["ff"], w, 1.5)
            mat(p + "mlp.down", w, l["mlp"]["ff"], loud)
            vec(p + "mlp.act", r.standard_normal(2))
    norm("final.norm")
    return W


def lively(cfg, seed):
    """Weights of a model that does not just repeat a token when it generates: loud layers, no preference among the tokens."""
    W = weights(cfg, seed, loud=8.0)
    W["final.norm.b"] = np.zeros_like(W["final.norm.b"])
    return W


OUT = {"retention": ["mix.o"], "left": ["mix.left.o"], "right": ["mix.right.o"], "ff": ["mlp.down"]}


def only(W, *keep):
    """A one-layer model's weights with the output projections of all sublayers but these at zero."""
    gone = {f"l0.{n}" for k, names in OUT.items() if k not in keep for n in names}
    return {n: np.zeros_like(v) if n in gone else v for n, v in W.items()}


# ── one token that stands out ───────────────────────────────────────────────
MARK, PLAIN = 0, 1


def _marker_embedding(W):
    """The first two coordinates of the mixer's input: whether the token is the marker, and one."""
    e = W["embed"]
    e[:, 0], e[:, 1] = 0.0, 9.0
    e[MARK, 0] = 9.0
    W["l0.norm1"][:2], W["l0.norm1.b"][:2], W["l0.norm1.alpha"] = 1.0, 0.0, np.float32(1.0)


def marker_attention(window, keep, heads=6, kv_heads=2, conv=3):
    """Every query looks for the marker token along a coordinate that is not rotated: a visible marker takes all of the attention, an
    invisible one leaves a broad mixture. The convolution leaves that coordinate alone."""
    cfg = config([parallel(left(heads=heads, kv_heads=kv_heads, dim=18, vdim=14, rot=8, window=window, keep=keep, conv=conv, softcap=25.0, scale=0.25), ff=None)], width=64)
    W = only(weights(cfg, seed=21), "left")
    _marker_embedding(W)
    p = "l0.mix.left."
    for n, H in (("q", heads), ("k", kv_heads)):
        W[p + n].reshape(H, 18, -1)[:, 17] = 0.0
        W[p + n + ".b"].reshape(H, 18)[:, 17] = 0.0
        W[p + n + ".conv"].reshape(H, 18, -1)[:, 17] = np.eye(conv)[-1]
    W[p + "q"].reshape(heads, 18, -1)[:, 17, 1] = 30.0
    W[p + "k"].reshape(kv_heads, 18, -1)[:, 17, 0] = 4.0
    return cfg, {n: bf16(v) for n, v in W.items()}


def marker_state(kind, heads=3):
    """Only the marker writes into the states, which keep it for good: without it every later output is another one."""
    if kind == "retention":
        cfg = config([retention(heads=heads, dim=18, vdim=12, rot=10, decay=[1.0] * heads)], width=64)
        W = weights(cfg, seed=22)
        _marker_embedding(W)
        k, q = (W["l0.mix." + n].reshape(heads, 18, -1) for n in "kq")
        k[:], k[:, 17, 0] = 0.0, 1.0
        q[:, 17], q[:, 17, 1] = 0.0, 4.0
    else:
        cfg = config([parallel(b=right(heads=heads, dim=18, vdim=12), ff=None)], width=64)
        W = only(weights(cfg, seed=22), "right")
        _marker_embedding(W)
        f = W["l0.mix.right.f"]
        f[:], f[:, 0] = 0.0, -50.0
        W["l0.mix.right.f.b"][:] = 25.0
    return cfg, {n: bf16(v) for n, v in W.items()}
