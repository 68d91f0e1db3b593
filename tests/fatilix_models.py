"""Small Fatilix configurations and weights for the tests, made here (not by the package's synthetic builder), so that every
size differs from every other where the design allows it. Weights are bf16-representable float32 arrays."""
import copy

import numpy as np

from plan_models import bf16, error, tokens  # noqa: F401  (the tests take them from here)


def temp(coef=0.4, every=19):
    return {"coef": coef, "every": every}


def shared_kv(heads=6, kv_heads=2, dim=20, scale=None, q_temp=True, mlp=True):
    """Keys that are the values."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or 1.3 * dim ** -0.5}
    return layer("attention", m, q_temp, moe() if mlp is True else mlp)


def biased(heads=6, kv_heads=3, dim=18, vdim=26, bias_max=60, rows=12, scale=None, q_temp=True, mlp=True):
    """A bias by distance. rows is no entry of the configuration: the table's shape tells it."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5, "bias_max": bias_max, "_rows": rows}
    return layer("attention_2", m, q_temp, dense() if mlp is True else mlp)


def layer(kind, mixer, q_temp, mlp):
    if q_temp:
        mixer["q_temp"] = temp() if q_temp is True else q_temp
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def dense(ff=52):
    return {"kind": "dense", "ff": ff}


def moe(experts=10, top=3, groups=(5, 2), ff=36, shared=28, scale=1.7):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    d = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def config(layers, vocab=150, width=88, eps=1e-5, scale=0.7, mult=0.6, max_positions=600):
    return {"architecture": "Fatilix", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "residual_mult": mult, "layers": layers}


def varied():
    """Every layer different: either attention with either feed-forward or none, groups of one to nine query heads, values
    smaller and larger than keys, odd sizes, bias tables of a few and of many rows, one expert, one group, every group kept."""
    return config([
        shared_kv(heads=6, kv_heads=2, dim=36, q_temp=temp(0.9, 7), mlp=dense(70)),
        biased(heads=6, kv_heads=2, dim=20, vdim=28, bias_max=90, rows=14, q_temp=temp(0.2, 31), mlp=None),
        biased(heads=9, kv_heads=1, dim=16, vdim=6, bias_max=6, rows=4, mlp=moe(experts=12, top=5, groups=(3, 2), ff=20, shared=None, scale=0.5)),
        shared_kv(heads=5, kv_heads=5, dim=9, mlp=moe(experts=1, top=1, groups=None, ff=50, shared=12)),
        shared_kv(heads=1, kv_heads=1, dim=50, q_temp=None, mlp=None),
        biased(heads=2, kv_heads=2, dim=44, vdim=17, bias_max=400, rows=33, q_temp=temp(1.5, 64), mlp=dense(33)),
        shared_kv(heads=18, kv_heads=1, dim=24, mlp=moe(experts=33, top=4, groups=(11, 4), ff=7, shared=90, scale=3.0)),
        biased(heads=1, kv_heads=1, dim=6, vdim=34, bias_max=17, rows=32, mlp=moe(experts=8, top=8, groups=(4, 4), ff=14, shared=5, scale=1.0)),
    ], vocab=153, width=90)


def weights(cfg, seed=0, sharp=1.0, loud=1.0):
    """Random weights; `sharp` scales the queries, so that attention concentrates on few keys; `loud` what the layers add to the
    stream."""
    r = np.random.default_rng(seed)
    W = {}

    def mat(name, n, k, gain=1.0):
        W[name] = bf16(r.standard_normal((n, k)) * gain / np.sqrt(k))

    def vec(name, v):
        W[name] = bf16(np.asarray(v, np.float32))

    w = cfg["width"]
    mat("embed", cfg["vocab"], w, 2.0 * np.sqrt(w))
    mat("pos", cfg["max_positions"], w, 0.8 * np.sqrt(w))
    for i, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], f"l{i}."
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        vec(p + "norm1", loud - 1 + 0.3 * r.standard_normal(w))
        mat(p + "mix.q", H * D, w)
        mat(p + "mix.k", G * D, w)
        if l["type"] == "attention":
            vec(p + "mix.q.norm", sharp * (1 + 0.3 * r.standard_normal(D)))
            vec(p + "mix.k.norm", 1 + 0.3 * r.standard_normal(D))
        else:
            mat(p + "mix.v", G * V, w)
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
                vec(p + f"mix.{n}.b", 0.7 * r.standard_normal(rows))
            vec(p + "mix.rel", 1.2 * r.standard_normal((m["_rows"], H)))
        vec(p + "mix.sink", 1.0 + r.standard_normal(H))
        mat(p + "mix.g", H * V, w, 0.6)
        mat(p + "mix.o", w, H * V)
        if not f:
            continue
        vec(p + "norm2", loud - 1 + 0.3 * r.standard_normal(w))
        if f["kind"] == "dense":
            mat(p + "mlp.up", f["ff"], w)
            mat(p + "mlp.down", w, f["ff"])
            continue
        E = f["router"]["experts"]
        mat(p + "mlp.router", E, w)
        vec(p + "mlp.correction", 0.6 / E * r.standard_normal(E) - 0.3 / E)   # some choice scores are negative
        for tag, ff in [(f"mlp.e{e}.", f["expert"]["ff"]) for e in range(E)] + ([("mlp.shared.", f["shared"]["ff"])] if f.get("shared") else []):
            mat(p + tag + "gate", ff, w)
            mat(p + tag + "up", ff, w)
            mat(p + tag + "down", w, ff)
    vec("final.norm", 0.3 * r.standard_normal(w))
    mat("head", cfg["vocab"], w)
    return W


def spelled(cfg):
    """For the restatement: what a configuration may leave out, as values that change nothing."""
    cfg = copy.deepcopy(cfg)
    for l in cfg["layers"]:
        l["mixer"].setdefault("q_temp", temp(0.0, 1))
        r = (l["mlp"] or {}).get("router")
        if r:
            r.setdefault("groups", {"count": 1, "keep": 1})
            r.setdefault("scale", 1.0)
    return cfg


def silent(W, *norms):
    """The sublayers of these norms add nothing to the stream."""
    return {n: np.full_like(v, -1.0) if n in norms else v for n, v in W.items()}


# ── one token that stands out ───────────────────────────────────────────────
MARK, PLAIN = 0, 1


def marker(kind, heads=6, kv_heads=2, sink=2.0):
    """Every query looks for the marker token: a marker takes most of the attention, without one the mixture is broad and the sink
    takes its part. Only the marker's keys have the coordinate that the queries ask for."""
    make = shared_kv if kind == "attention" else biased
    cfg = config([make(heads=heads, kv_heads=kv_heads, dim=18, scale=0.6, mlp=None)], width=64)
    W = weights(cfg, seed=21, loud=2.0)
    e = W["embed"]
    e[:, 0], e[:, 1] = 0.0, 4.0
    e[MARK, 0] = 40.0
    W["pos"][:, :2] = 0.0
    q, k = W["l0.mix.q"].reshape(heads, 18, -1), W["l0.mix.k"].reshape(kv_heads, 18, -1)
    q[:, 17], k[:, 17] = 0.0, 0.0
    q[:, 17, 1], k[:, 17, 0] = 6.0, 1.0
    if kind == "attention":
        W["l0.mix.q.norm"][17] = W["l0.mix.k.norm"][17] = 1.0
    else:
        W["l0.mix.q.b"].reshape(heads, 18)[:, 17] = 0.0
        W["l0.mix.k.b"].reshape(kv_heads, 18)[:, 17] = 0.0
    W["l0.mix.sink"][:] = sink
    return cfg, {n: bf16(v) for n, v in W.items()}


def one_distance(at, bias_max=200, rows=20, heads=4, kv_heads=2):
    """The bias alone says where a head looks: the row of one distance stands out, the others are low, keys are all alike."""
    from oracle import fatilix as L

    cfg = config([biased(heads=heads, kv_heads=kv_heads, dim=12, vdim=22, bias_max=bias_max, rows=rows, scale=1e-3, mlp=None)], width=64)
    W = weights(cfg, seed=23, loud=2.0)
    W["l0.mix.rel"][:] = -6.0
    W["l0.mix.rel"][L.bucket(at, rows, bias_max)] = 6.0
    W["l0.mix.sink"][:] = 0.0
    return cfg, {n: bf16(v) for n, v in W.items()}
