"""CPU side of the Revelix tests: the restatement's mechanisms against hand-made cases, planted mistakes that the GPU tests'
inputs must expose, and the configuration reader of the library."""
import copy
import ctypes as C
import json
import math

import numpy as np
import pytest

import revelix_models as M
from oracle import revelix as L
from sapient_b200 import _lib, synth
from sapient_b200.engine import ForwardEngine


# ── the restatement ─────────────────────────────────────────────────────────
def test_norm_has_no_statistics():
    W = {"n": np.array([2.0, 3.0]), "n.b": np.array([0.5, -1.0]), "n.alpha": np.array(0.5)}
    assert np.allclose(L.tanh_norm(np.array([[1.0, -4.0]]), W, "n"), [[2 * math.tanh(0.5) + 0.5, 3 * math.tanh(-2.0) - 1]])


def test_activation_is_smooth_at_zero_and_odd_nowhere():
    p, q = 0.3, -0.7
    ap, an = math.log1p(math.exp(p)), 0.5 + math.log1p(math.exp(q))
    got = L.xielu(np.array([2.0, -1.0, 0.0, 1e-9, -1e-9]), p, q)
    assert np.allclose(got, [ap * 4 + 1, an * (math.exp(-1) - 1 + 1) - 0.5, 0, 5e-10, -5e-10], rtol=1e-9, atol=1e-15)


def test_rotations():
    x = np.array([[1.0, 0.0, 0.0, 0.0, 5.0]])
    rot = {"base": 100.0, "dims": 4}
    assert np.allclose(L.rotate(x, np.array([3]), rot, False)[0], [np.cos(3), 0, np.sin(3), 0, 5])
    assert np.allclose(L.rotate(x, np.array([3]), rot, True)[0], [np.cos(3), np.sin(3), 0, 0, 5])
    y = L.rotate(np.array([[0.0, 0.0, 0.0, 1.0]]), np.array([3]), rot, True)
    assert np.allclose(y[0], [0, 0, -np.sin(0.3), np.cos(0.3)])            # 3 * 100^(-2/4)


def test_stretched_frequencies():
    dims, base, original = 16, 1000.0, 500
    s = dict(factor=4.0, original=original, fast=10.0, slow=1.0)
    f, g = L.frequencies(dims, base), L.stretched_frequencies(dims, base, **s)
    turns = original * f / (2 * math.pi)
    assert np.allclose(g[0], f[0]) and np.allclose(g[-1], f[-1] / 4)
    assert np.all(np.diff(g / f) <= 1e-12) and np.allclose((g / f)[turns < 0.5], 0.25)
    x = np.array([[1.0, 0.0]])
    assert np.allclose(L.rotate(x, np.array([0]), {"base": base, "dims": 2, "scaling": s}, True)[0], [0.1 * math.log(4) + 1, 0])
    # both ends of the ramp at one pair: a step, not a division by zero
    assert np.isfinite(L.stretched_frequencies(4, 10.0, factor=2.0, original=10, fast=1e6, slow=1e5)).all()


def test_convolution_looks_back_only():
    u = np.array([[1.0], [10.0], [100.0], [1000.0]])
    assert np.allclose(L.short_conv(u, np.array([[3.0, 2.0, 1.0]]))[:, 0], [1, 12, 123, 1230])
    assert np.allclose(L.short_conv(u, np.array([[0.5]])), 0.5 * u)


def test_window_counts_the_token_itself_and_keeps_the_first():
    assert L.kept_window_mask(7, 2, 3)[6].tolist() == [True, True, True, False, False, True, True]
    assert L.kept_window_mask(7, 2, 3)[1].tolist() == [True, True] + 5 * [False]
    assert np.array_equal(L.kept_window_mask(4, 1, 0), np.eye(4, dtype=bool))


def test_weights_are_mixed_without_the_sink():
    w = L.sink_weights(np.log(np.array([[[1.0, 2.0]], [[3.0, 1.0]]])), np.log(np.array([1.0, 4.0])))
    assert np.allclose(w, [[[0.25, 0.5]], [[0.375, 0.125]]])
    assert np.allclose(L.mixed_heads(w, np.array([[1.0, 2.0], [0.0, -1.0]])), [[[1.0, 0.75]], [[-0.375, -0.125]]])


def test_scans():
    r = np.random.default_rng(2)
    q, k, v = r.standard_normal((2, 5, 3)), r.standard_normal((2, 5, 3)), r.standard_normal((2, 5, 4))
    d = np.array([0.5, 1.0])
    want = sum(d[:, None] ** (4 - j) * np.einsum("hd,hd->h", q[:, 4], k[:, j])[:, None] * v[:, j] for j in range(5))
    assert np.allclose(L.decaying_sum(q, k, v, d)[:, 4], want)
    f = r.uniform(0, 1, (2, 5, 3))
    want = sum(np.einsum("hd,hd->h", q[:, 4], (1 - f[:, j]) * np.prod(f[:, j + 1:], axis=1))[:, None] * v[:, j] for j in range(5))
    assert np.allclose(L.gated_sum(q, f, v)[:, 4], want)


def test_forget_gate_keeps_its_bound():
    W = {"f": np.zeros((3, 2)), "f.b": np.array([-50.0, 0.0, 50.0]), "lower": np.array([0.25, 0.5, 0.0])}
    assert np.allclose(L.forget(np.zeros((1, 2)), W, ""), [[0.25, 0.75, 1.0]])


def test_last_position_does_not_depend_on_later_tokens():
    cfg = M.varied()
    W = M.weights(cfg)
    ids = M.tokens(cfg, 40)
    assert np.allclose(L.forward(cfg, W, ids)[0][:25], L.forward(cfg, W, ids[:25])[0])


# ── the GPU tests' inputs expose mistakes ───────────────────────────────────
MASK, ROT, CONV, SINK, DECAY, GATED, FORGET, XIELU, RET, SCAN_RMS, ATT = (L.kept_window_mask, L.rotate, L.short_conv, L.sink_weights, L.decaying_sum, L.gated_sum, L.forget,
                                                                        L.xielu, L.retention, L.rms, L.attention)


def lost(f, at):                                              # a state that starts again at a token
    return lambda *x: np.concatenate([f(*[y[:, :at] if np.ndim(y) > 1 else y for y in x]), f(*[y[:, at:] if np.ndim(y) > 1 else y for y in x])], 1)


def conv_cut(u, w):                                           # a portion that forgets what came before it
    return np.concatenate([CONV(u[:70], w), CONV(u[70:], w)])


def plain_rotation(x, pos, rot, pairs):
    return ROT(x, pos, {"base": rot["base"], "dims": rot["dims"]}, pairs)


def no_magnitude(x, pos, rot, pairs):
    return ROT(x, pos, rot, pairs) / np.where(np.arange(x.shape[-1]) < rot["dims"], L.magnitude(rot.get("scaling")), 1.0)


def cap_before_scale(s, cap):
    return np.clip(s, -cap, cap)


def sink_mixed(weights, talk):
    return np.einsum("hg,gij->hij", talk, weights) / np.maximum(weights.sum(-1, keepdims=True), 1e-9)


MISTAKES = {
    "window one wider": dict(kept_window_mask=lambda T, s, k: MASK(T, s + 1, k)),
    "window one narrower": dict(kept_window_mask=lambda T, s, k: MASK(T, max(1, s - 1), k)),
    "one kept key more": dict(kept_window_mask=lambda T, s, k: MASK(T, s, k + 1)),
    "one kept key less": dict(kept_window_mask=lambda T, s, k: MASK(T, s, max(0, k - 1))),
    "nothing kept": dict(kept_window_mask=lambda T, s, k: MASK(T, s, 0)),
    "pairs the other way": dict(rotate=lambda x, p, r, pairs: ROT(x, p, r, not pairs)),
    "positions one off late": dict(rotate=lambda x, p, r, pairs: ROT(x, np.where(p > 60, p + 1, p), r, pairs)),
    "frequencies not stretched": dict(rotate=plain_rotation),
    "no magnitude": dict(rotate=no_magnitude),
    "convolution reversed": dict(short_conv=lambda u, w: CONV(u, w[:, ::-1])),
    "convolution forgets": dict(short_conv=conv_cut),
    "no convolution": dict(short_conv=lambda u, w: u * w[:, -1]),
    "no cap": dict(capped=lambda s, cap: s),
    "cap as a clip": dict(capped=cap_before_scale),
    "no sink": dict(sink_weights=lambda s, k: SINK(s, np.full_like(k, -1e9))),
    "heads not mixed": dict(mixed_heads=lambda w, t: w),
    "mixed the other way": dict(mixed_heads=lambda w, t: np.einsum("gh,gij->hij", t, w)),
    "sink mixed": dict(mixed_heads=sink_mixed),
    "retention lost": dict(decaying_sum=lost(DECAY, 70)),
    "keys not scaled": dict(decaying_sum=lambda q, k, v, d: DECAY(q, k * 1.3, v * 1.3, d ** 2)),
    "gated state lost": dict(gated_sum=lost(GATED, 70)),
    "key is the kept share": dict(gated_sum=lambda q, f, v: GATED(q, 1 - f, v)),
    "no lower bound": dict(forget=lambda h, W, p: FORGET(h, {**W, p + "lower": np.zeros_like(W[p + "lower"])}, p)),
    "gate without bias": dict(forget=lambda h, W, p: FORGET(h, {**W, p + "f.b": np.zeros_like(W[p + "f.b"])}, p)),
    "no silu": dict(silu=lambda z: z),
    "sigmoid gate": dict(silu=L.sigmoid),
    "activation's numbers swapped": dict(xielu=lambda z, p, q: XIELU(z, q, p)),
    "activation without softplus": dict(xielu=lambda z, p, q: z / 2 + np.where(z > 0, p * z * z, (0.5 + q) * (np.expm1(np.minimum(z, 0)) - np.minimum(z, 0)))),
    "head outputs not normed": dict(rms=lambda x, eps: x),
    "norm over all heads": dict(rms=lambda x, eps: x / np.sqrt(np.mean(x * x, axis=(0, 2), keepdims=True) + eps)),
    "one branch alone": dict(parallel=lambda h, W, p, m, eps, pos: ATT(h, W, p + "left.", m["left"], eps, pos) * m["left_scale"]),
    "scales left out": dict(attention=lambda h, W, p, m, eps, pos: ATT(h, W, p, m, eps, pos) * 1.3),
}


@pytest.mark.parametrize("name", MISTAKES)
def test_planted_mistakes_show(name):
    cfg = M.varied()
    W = M.weights(cfg, seed=2, sharp=2.0)
    ids = M.tokens(cfg, 90)
    want = L.forward(cfg, W, ids)[0]
    mixers = dict(L.MIXERS)
    old = {k: getattr(L, k) for k in MISTAKES[name]}
    try:
        for k, f in MISTAKES[name].items():
            setattr(L, k, f)
            if k in L.MIXERS:
                L.MIXERS[k] = f
        e = M.error(L.forward(cfg, W, ids)[0], want)
    finally:
        for k, f in old.items():
            setattr(L, k, f)
        L.MIXERS.update(mixers)
    assert np.max(e) > 0.1, float(np.max(e))


@pytest.mark.parametrize("window,keep", [(16, 0), (64, 0), (16, 9), (33, 20)])
def test_marker_places_are_sharp(window, keep):
    cfg, W = M.marker_attention(window, keep)
    mask = ("layers", 0, "mixer", "left", "mask")
    for at, key in ((keep + 4, "size"), (keep, "keep_first")):  # a key behind the kept ones, and the first that is not kept
        n = at + window + 6
        ids = (1 + np.arange(n) % 50).astype(np.uint32)
        ids[at] = M.MARK
        other = copy.deepcopy(cfg)
        m = other
        for k in mask:
            m = m[k]
        m[key] += 1
        e = M.error(L.forward(other, W, ids)[0], L.forward(cfg, W, ids)[0])
        assert e[at + window] > 0.25 and np.all(e[:at + window] < 1e-6)


@pytest.mark.parametrize("kind", ["retention", "forget"])
def test_marked_states_are_sharp(kind):
    cfg, W = M.marker_state(kind)
    ids = (1 + np.arange(300) % 50).astype(np.uint32)
    with_it = ids.copy()
    with_it[4] = M.MARK
    e = M.error(L.forward(cfg, W, with_it)[0], L.forward(cfg, W, ids)[0])
    assert np.all(e[4:] > 0.25) and np.all(e[:4] < 1e-6)


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
    assert st == _lib.SP_OK and (d.arch, d.n_layers, d.hidden, d.vocab) == (2, 8, 90, 153)
    assert ForwardEngine.arch_block("Revelix") == 2
    plain = M.varied()
    del plain["logit_scale"], plain["layers"][0]["mlp"]
    assert create(plain)[0] == _lib.SP_OK
    m = plain["layers"][0]["mixer"]
    del m["left_scale"], m["right_scale"], m["left"]["mask"], m["left"]["softcap"], m["left"]["conv"], m["left"]["rot"]["scaling"]
    assert create(plain)[0] == _lib.SP_OK


LEFT = ["layers", 0, "mixer", "left"]


@pytest.mark.parametrize("path,value,word", [
    (["vocab"], None, "vocab"), (["width"], 0, "width"), (["norm"], None, "norm"), (["layers"], [], "layers"), (["logit_scale"], "x", "logit_scale"),
    (["layers", 1, "type"], "attention", "type"), (["layers", 0, "mixer", "right"], None, "right"), (["layers", 0, "mixer", "left_scale"], "x", "left_scale"),
    (["layers", 0, "mixer", "right_scale"], "x", "right_scale"), (["layers", 0, "mixer", "right", "dim"], 1000, "dim"), (LEFT + ["kv_heads"], 4, "kv_heads"),
    (LEFT + ["conv"], 0, "conv"), (LEFT + ["conv"], 33, "conv"), (LEFT + ["softcap"], 0, "softcap"), (LEFT + ["mask", "size"], 0, "size"),
    (LEFT + ["mask", "keep_first"], -1, "keep_first"), (LEFT + ["scale"], None, "scale"), (LEFT + ["rot", "dims"], 22, "rot"), (LEFT + ["rot", "dims"], 7, "rot"),
    (LEFT + ["rot", "scaling", "factor"], 0, "scaling"), (LEFT + ["rot", "scaling", "slow"], None, "slow"), (["layers", 1, "mixer", "decay"], [0.5], "decay"),
    (["layers", 1, "mixer", "rot"], None, "rot"), (["layers", 1, "mixer", "rot", "base"], None, "base"), (["layers", 1, "mixer", "heads"], 1.5, "heads"),
    (["layers", 0, "mlp", "kind"], "moe", "kind"), (["layers", 0, "mlp", "ff"], None, "ff")], ids=str)
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
    cfg = synth.revelix_config(layers=["retention", "parallel", "retention"], width=48, heads=4, kv_heads=2, dim=8, vdim=12, state_heads=3, state_dim=10, state_vdim=6,
                               retention_heads=5, retention_dim=6, retention_vdim=14, window=9, keep_first=2, ff=20, vocab=30, conv=4)
    a = {k: int(v.numel()) for k, v in synth.revelix_weights(cfg, 0).items()}
    assert a == {k: int(np.size(v)) for k, v in M.weights(cfg).items()}
