"""Small Lepalorn configurations and weights for the tests, made here (not by the package's synthetic builder), so that
every size differs from every other where the design allows it. Weights are bf16-representable float32 arrays."""
import numpy as np


def bf16(x):
    """float32 values rounded to the nearest bfloat16 (ties to even)."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).view(np.float32).reshape(np.shape(x))


def mixer(heads=3, dim=24, rot=8, vdim=20, rank=40, window=13, scale=None, base=700.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale or 1.3 * (dim + rot) ** -0.5,
         "mask": {"size": window}, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def moe(experts=5, top=2, ff=36, limit=0.9, shared=(28, 0.6)):
    d = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared:
        d["shared"] = {"ff": shared[0], "limit": shared[1]}
    return d


def config(layers, vocab=150, width=88, eps=1e-5, scale=0.7):
    return {"architecture": "Lepalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


def varied():
    """Every layer different: own and borrowed latents out of order, with and without a feed-forward or shared expert,
    windows from one key to more than any test's context, one expert, one head, odd widths."""
    a = dict(rank=40, rot=8, base=700.0)
    b = dict(rank=72, rot=6, base=90.0)
    return config([
        (mixer(heads=3, dim=24, vdim=20, window=13, **a), moe()),
        (mixer(heads=5, dim=9, vdim=33, window=29, **b), moe(experts=7, top=3, ff=20, limit=0.4, shared=None)),
        (mixer(heads=2, dim=40, vdim=8, window=5, kv_from=0, **a), None),
        (mixer(heads=1, dim=16, vdim=50, window=64, kv_from=1, **b), moe(experts=1, top=1, ff=50, limit=2.0)),
        (mixer(heads=17, dim=4, vdim=4, window=1, kv_from=0, **a), moe(experts=33, top=4, ff=7, shared=(90, 0.3))),
        (mixer(heads=4, dim=12, vdim=12, rank=16, rot=2, base=5.0, window=4000), moe(shared=(12, 1.5))),
    ], vocab=151, width=90)


def uniform(n=2, **kw):
    return config([(mixer(**kw), moe()) for _ in range(n)])


def weights(cfg, seed=0, sharp=1.0):
    """Random weights; `sharp` scales the queries, so that attention concentrates on few keys."""
    r = np.random.default_rng(seed)
    W = {}

    def mat(name, n, k, gain=1.0):
        W[name] = bf16(r.standard_normal((n, k)) * gain / np.sqrt(k))

    def num(name, v):
        W[name] = bf16(np.asarray(v, np.float32))

    w = cfg["width"]
    mat("embed", cfg["vocab"], w, 2.0 * np.sqrt(w))
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        num(p + "norm1", 0.6 + 0.1 * i)
        mat(p + "mix.q", H * (D + R), w, sharp)
        if "kv_from" not in m:
            mat(p + "mix.dkv", K + R, w)
            num(p + "mix.dkv.norm", 1 + 0.3 * r.standard_normal(K))
        mat(p + "mix.uk", H * D, K)
        mat(p + "mix.uv", H * V, K)
        mat(p + "mix.g", H, w)
        mat(p + "mix.o", w, H * V)
        if f:
            num(p + "norm2", 0.9 - 0.1 * i)
            E = f["router"]["experts"]
            mat(p + "mlp.router", E, w, 2.0)
            num(p + "mlp.router.b", 0.5 * r.standard_normal(E))
            parts = [(f"mlp.e{e}.", f["expert"]["ff"]) for e in range(E)]
            if "shared" in f:
                parts.append(("mlp.shared.", f["shared"]["ff"]))
                mat(p + "mlp.shared.sg", 1, w)
            for tag, ff in parts:
                mat(p + tag + "gate", ff, w)
                mat(p + tag + "up", ff, w)
                mat(p + tag + "down", w, ff)
        c = 0.4 * r.standard_normal(i + 2)
        c[-1] += 1
        num(p + "dwa", c)
    num("final.norm", 1.2)
    mat("head", cfg["vocab"], w)
    return W


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n).astype(np.uint32)


def error(got, want):
    """Root mean square of the difference over the vocabulary, mean taken off, relative to the spread of the logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.std(want)


def boundary_logits(z, k):
    """Gap between the k-th and the next logit of each row: how close the choice of experts is."""
    s = -np.sort(-z, axis=-1)
    return s[:, k - 1] - s[:, k] if k < z.shape[1] else np.full(len(z), np.inf)
