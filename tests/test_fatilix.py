"""CPU side of the Fatilix tests: the restatement's mechanisms against hand-made cases, planted mistakes that the GPU tests'
inputs must expose, and the configuration reader of the library."""
import copy
import ctypes as C
import json
import math

import numpy as np
import pytest

import fatilix_models as M
from oracle import fatilix as L
from sapient_b200 import _lib, synth
from sapient_b200.engine import ForwardEngine


# ── the restatement ─────────────────────────────────────────────────────────
def test_offset_norm_and_residual():
    x = np.array([[3.0, 4.0]])
    want = x / math.sqrt(12.5 + 0.5) * np.array([1.5, 0.0])
    assert np.allclose(L.offset_norm(x, np.array([0.5, -1.0]), 0.5), want)
    assert np.allclose(L.residual(np.ones((1, 2)), x, np.array([0.5, -1.0]), 0.5, 0.7), 1 + 0.7 * want)


def test_embedding_adds_positions_unscaled():
    W = {"embed": np.arange(6.0).reshape(3, 2), "pos": np.array([[10.0, 20], [30, 40], [50, 60]])}
    assert np.allclose(L.embedding(np.array([2, 0]), W, 0.5), [[12, 22.5], [30, 40.5]])


def test_temperature_steps():
    t = L.temperature(np.arange(12), 0.5, 4)
    assert np.allclose(t, 1 + 0.5 * np.log([1, 1, 1, 2, 2, 2, 2, 3, 3, 3, 3, 4]))


def test_buckets():
    rows, far = 8, 64                                          # exact up to 3, then 4 rows over a factor of 16: one per doubling
    got = [L.bucket(n, rows, far) for n in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)]
    assert got == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    b = L.distance_bias(np.arange(16.0).reshape(8, 2), 64, 10)
    assert b.shape == (2, 10, 10) and b[1, 9, 1] == 2 * 5 + 1 and b[0, 5, 5] == 0 and b[1, 5, 4] == 3


def test_sink_takes_its_part_and_is_not_mixed():
    w = L.sink_weights(np.log(np.array([[[1.0, 2.0, 5.0]]])), np.log(np.array([2.0])))
    assert np.allclose(w, [[[0.1, 0.2, 0.5]]])
    w = L.sink_weights(np.array([[[-np.inf, 0.0]]]), np.array([500.0]))
    assert np.allclose(w, 0) and np.isfinite(w).all()


def test_values_are_the_projected_keys():
    """One token: the mixture is its projected key without norm, times the share that the sink leaves."""
    cfg = M.config([M.shared_kv(heads=2, kv_heads=1, dim=4, q_temp=None, mlp=None)], width=6)
    W = {k: np.asarray(v, np.float64) for k, v in M.weights(cfg).items()}
    W["l0.mix.o"] = np.eye(6, 8)
    W["l0.mix.sink"][:] = -1e9
    h = np.random.default_rng(1).standard_normal((1, 6))
    o = L.attention(h, W, "l0.mix.", cfg["layers"][0]["mixer"] | {"q_temp": {"coef": 0.0, "every": 1}}, 1e-5, np.arange(1))
    gate = 1 / (1 + np.exp(-(h @ W["l0.mix.g"].T)))
    assert np.allclose(o[0], (np.tile(h @ W["l0.mix.k"].T, 2) * gate)[0, :6])


def route(scores, correction, **r):
    """Router logits chosen so that the scores are the given ones."""
    s = np.asarray(scores, np.float64)
    W = {"router": np.log(s)[:, None], "correction": np.asarray(correction, np.float64)}
    pick, w = L.route(np.ones((1, 1)), W, "", r)
    return pick[0].tolist(), w[0]


def test_choice_by_groups_and_weights_without_the_correction():
    s = [0.30, 0.05, 0.20, 0.22, 0.10, 0.13]
    assert route(s, np.zeros(6), top=3, groups={"count": 3, "keep": 2}, scale=2.0)[0] == [0, 3, 2]
    pick, w = route(s, [0, 0, -0.5, -0.5, 0, 0], top=3, groups={"count": 3, "keep": 2}, scale=2.0)
    assert pick == [0, 5, 4] and np.allclose(w, 2 * np.array([0.30, 0.13, 0.10]) / 0.53)
    # all of a kept group's scores may be negative: they still come before those of the groups that are not kept
    pick, _ = route(s, [-0.9, -0.9, -0.5, -0.5, -1.0, -1.0], top=4, groups={"count": 3, "keep": 2}, scale=1.0)
    assert pick == [3, 2, 0, 1]


def test_one_group_means_no_restriction():
    assert route([0.1, 0.4, 0.2, 0.3], np.zeros(4), top=2, groups={"count": 1, "keep": 1}, scale=1.0)[0] == [1, 3]


def test_last_position_does_not_depend_on_later_tokens():
    cfg = M.varied()
    W = M.weights(cfg)
    ids = M.tokens(cfg, 40)
    assert np.allclose(oracle(cfg, W, ids)[:25], oracle(cfg, W, ids[:25]))


# ── the GPU tests' inputs expose mistakes ───────────────────────────────────
def oracle(cfg, W, ids):
    return L.forward(M.spelled(cfg), W, ids)[0]


def changed(cfg, W, ids, patch):
    want = oracle(cfg, W, ids)
    old = {k: getattr(L, k) for k in patch}
    try:
        for k, f in patch.items():
            setattr(L, k, f)
        return M.error(oracle(cfg, W, ids), want)
    finally:
        for k, f in old.items():
            setattr(L, k, f)


BUCKET, TEMP, NORM, ROUTE, ATTN, ATTN2 = L.bucket, L.temperature, L.offset_norm, L.route, L.attention, L.attention_2


def weights_with_the_correction(h, W, p, r):
    pick, _ = ROUTE(h, W, p, r)
    w = np.take_along_axis(L.softmax(h @ W[p + "router"].T) + W[p + "correction"], pick, axis=-1)
    return pick, w / (w.sum(-1, keepdims=True) + 1e-20) * r["scale"]


def struck_out_as_zero(h, W, p, r):
    s = L.softmax(h @ W[p + "router"].T)
    choice = s + W[p + "correction"]
    pick = L.best(np.where(L.allowed_experts(choice, r["groups"]["count"], r["groups"]["keep"]), choice, 0.0), r["top"])
    w = np.take_along_axis(s, pick, axis=-1)
    return pick, w / w.sum(-1, keepdims=True) * r["scale"]


def normed_values(h, W, p, m, eps, pos):
    k = L.split_heads(h @ W[p + "k"].T, m["kv_heads"])
    q = L.rms(L.split_heads(h @ W[p + "q"].T, m["heads"]), eps) * W[p + "q.norm"] * L.temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"])[None, :, None]
    k = L.rms(k, eps) * W[p + "k.norm"]
    return L.output_gate(L.mix(q, k, k, 0.0, W, p, m), h, W, p) @ W[p + "o"].T


MISTAKES = {
    "bucket one late": dict(bucket=lambda n, rows, far: BUCKET(max(n - 1, 0), rows, far)),
    "bucket rounded": dict(bucket=lambda n, rows, far: n if n < rows // 2 else min(rows - 1, rows // 2 + round(math.log(n / (rows // 2)) / math.log(far / (rows // 2)) * (rows - rows // 2)))),
    "bias scaled": dict(distance_bias=lambda t, far, T: 0.2 * DISTANCE(t, far, T)),
    "no bias": dict(distance_bias=lambda t, far, T: 0.0),
    "no temperature": dict(temperature=lambda p, c, e: np.ones(len(p))),
    "temperature one late": dict(temperature=lambda p, c, e: TEMP(p - 1, c, e)),
    "temperature without floor": dict(temperature=lambda p, c, e: 1 + c * np.log((p + 1) / e + 1)),
    "no sink": dict(sink_weights=lambda s, k: L.softmax(s)),
    "no gate": dict(output_gate=lambda o, h, W, p: o),
    "sees the next key": dict(causal=lambda T: np.arange(T)[:, None] + 1 >= np.arange(T)[None, :]),
    "weight not from one": dict(offset_norm=lambda x, w, eps: L.rms(x, eps) * w),
    "no factor": dict(residual=lambda x, y, w, eps, mult: x + NORM(y, w, eps)),
    "positions scaled": dict(embedding=lambda ids, W, s: (W["embed"][ids] + W["pos"][: len(ids)]) * s),
    "positions one late": dict(embedding=lambda ids, W, s: W["embed"][ids] * s + W["pos"][1: len(ids) + 1]),
    "values normed": dict(attention=normed_values),
    "relu not squared": dict(squared_relu=lambda z: np.maximum(z, 0)),
    "no silu": dict(silu=lambda z: z),
    "all groups": dict(allowed_experts=lambda c, g, k: np.ones(c.shape, bool)),
    "one group more": dict(allowed_experts=lambda c, g, k: ALLOWED(c, g, min(g, k + 1))),
    "weights with the correction": dict(route=weights_with_the_correction),
    "struck out as zero": dict(route=struck_out_as_zero),
    "weights not scaled": dict(route=lambda h, W, p, r: ROUTE(h, W, p, r | {"scale": 1.0})),
}
DISTANCE, ALLOWED = L.distance_bias, L.allowed_experts


@pytest.mark.parametrize("name", MISTAKES)
def test_planted_mistakes_show(name):
    cfg = M.varied()
    W = M.weights(cfg, seed=2, sharp=2.0)
    e = changed(cfg, W, M.tokens(cfg, 90), MISTAKES[name])
    assert np.max(e) > 0.05, float(np.max(e))
    if name in ("no sink", "no gate", "no factor", "no temperature"):
        assert np.median(e) > 0.05


@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_markers_and_sinks_are_sharp(kind):
    cfg, W = M.marker(kind)
    ids = (1 + np.arange(300) % 50).astype(np.uint32)
    with_it = ids.copy()
    with_it[4] = M.MARK
    want = oracle(cfg, W, ids)
    e = M.error(oracle(cfg, W, with_it), want)
    assert np.all(e[4:] > 0.25) and np.all(e[:4] < 1e-9)
    W["l0.mix.sink"][:] = -30.0
    assert M.error(oracle(cfg, W, ids), want)[0] > 0.25


@pytest.mark.parametrize("at", [3, 9, 10, 40, 150, 260])
def test_one_distance_is_sharp(at):
    cfg, W = M.one_distance(at)
    ids = M.tokens(cfg, 280)
    first = next(n for n in range(at + 1) if L.bucket(n, 20, 200) == L.bucket(at, 20, 200))
    late = changed(cfg, W, ids, dict(bucket=lambda n, rows, far: BUCKET(max(n - 1, 0), rows, far)))
    assert late[first] > 0.25                                  # the first token that has a key in the bucket


# ── readers ─────────────────────────────────────────────────────────────────
def create(cfg, ctx=64):
    h, d = C.c_void_p(), ForwardEngine._run_desc(0, ctx, 1, 16, 0)
    st = _lib.lib().sp_cuda_engine_create_from_config(json.dumps(cfg).encode(), 30, C.byref(d), C.byref(h))
    if st == _lib.SP_OK:
        out = _lib.SpModelDesc()
        assert _lib.lib().sp_cuda_engine_desc(h, C.byref(out)) == _lib.SP_OK
        _lib.lib().sp_cuda_engine_destroy(h)
        return st, out
    return st, _lib.lib().sp_cuda_last_error().decode()


def test_configuration_is_read_from_the_file():
    st, d = create(M.varied())
    assert st == _lib.SP_OK and (d.arch, d.n_layers, d.hidden, d.vocab, d.max_ctx) == (2, 8, 90, 153, 64)
    assert ForwardEngine.arch_block("Fatilix") == 2
    assert create(M.varied(), ctx=5000)[1].max_ctx == 600    # no more positions than the table has


@pytest.mark.parametrize("path,value,word", [
    (["vocab"], None, "vocab"), (["width"], 0, "width"), (["norm"], None, "norm"), (["layers"], [], "layers"), (["max_positions"], 0, "max_positions"),
    (["residual_mult"], None, "residual_mult"), (["embedding"], None, "embedding"), (["layers", 1, "type"], "general_delta", "type"),
    (["layers", 0, "mixer", "vdim"], 9, "vdim"), (["layers", 0, "mixer", "kv_heads"], 4, "kv_heads"), (["layers", 1, "mixer", "bias_max"], None, "bias_max"),
    (["layers", 1, "mixer", "q_temp", "every"], 0, "every"), (["layers", 1, "mixer", "q_temp", "coef"], None, "coef"), (["layers", 1, "mixer", "scale"], "x", "scale"),
    (["layers", 0, "mlp", "kind"], "gated", "kind"), (["layers", 0, "mlp", "ff"], None, "ff"), (["layers", 2, "mlp", "expert"], None, "expert"),
    (["layers", 2, "mlp", "router", "groups", "count"], 5, "groups"), (["layers", 2, "mlp", "router", "groups", "keep"], 4, "keep"),
    (["layers", 2, "mlp", "router", "top"], 9, "top"), (["layers", 3, "mlp", "shared", "ff"], 0, "ff")])
def test_bad_configurations_are_named(path, value, word):
    cfg = copy.deepcopy(M.varied())
    at = cfg
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    st, msg = create(cfg)
    assert st == _lib.SP_ERR_ARG and word in msg, msg


def test_synthetic_builder_makes_the_same_tensors_as_the_tests():
    cfg = synth.fatilix_config(layers=["attention", "attention_2", "attention"], width=48, heads=4, kv_heads=2, dim=8, vdim=12, ff=20, experts=6, top=2,
                               groups=3, keep=2, expert_ff=10, shared_ff=14, vocab=30, max_positions=70, bias_max=40)
    a = {k: tuple(v.shape) for k, v in synth.fatilix_weights(cfg, 0, bias_rows=9).items()}
    cfg["layers"][1]["mixer"]["_rows"] = 9
    assert a == {k: tuple(np.shape(v)) for k, v in M.weights(cfg).items()}
