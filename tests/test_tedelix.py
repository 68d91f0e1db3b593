"""CPU side of the Tedelix tests: the restatement's mechanisms against hand-made cases, planted mistakes that the GPU tests'
inputs must expose, and the configuration reader of the library."""
import ctypes as C
import json

import numpy as np
import pytest

import tedelix_models as M
from oracle import tedelix as L
from sapient_b200 import _lib, synth
from sapient_b200.engine import ForwardEngine


# ── the restatement ─────────────────────────────────────────────────────────
def test_rotation_pairs_halves_and_passes_the_rest():
    x = np.array([[1.0, 0.0, 0.0, 0.0, 5.0]])
    y = L.rotate_halves(x, np.array([3]), 4, 100.0)
    assert np.allclose(y[0], [np.cos(3), 0, np.sin(3), 0, 5])
    y = L.rotate_halves(np.array([[0.0, 1.0, 0.0, 0.0]]), np.array([3]), 4, 100.0)
    assert np.allclose(y[0], [0, np.cos(0.3), 0, np.sin(0.3)])            # 3 * 100^(-2/4)


def test_rotated_values_depend_on_the_distance_only():
    """With one visible key its value comes back turned by the distance, wherever the pair stands."""
    v = np.random.default_rng(0).standard_normal((1, 8))
    at = lambda j, i: L.turned_back(L.rotated_values(v, np.array([j]), 50.0), np.array([i]), 50.0)  # noqa: E731
    assert np.allclose(at(7, 7), v) and np.allclose(at(3, 9), at(103, 109)) and not np.allclose(at(3, 9), at(3, 10))


def test_window_counts_the_token_itself():
    assert L.window_mask(6, 3)[5].tolist() == [False, False, False, True, True, True]
    assert np.array_equal(L.window_mask(4, 1), np.eye(4, dtype=bool))


def test_heads_share_cached_heads_in_runs():
    cfg = M.config([M.attention(heads=4, kv_heads=2, dim=4, vdim=2, rot=0, window=9, ff=None)], width=12)
    W = M.weights(cfg)
    h = np.random.default_rng(1).standard_normal((5, 12))
    W["l0.mix.q"] = np.tile(W["l0.mix.q"][:4], (4, 1))
    o = L.attention(h, W, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5, np.arange(5)).reshape(5, 4, 2)
    assert np.allclose(o[:, 0], o[:, 1]) and np.allclose(o[:, 2], o[:, 3]) and not np.allclose(o[:, 1], o[:, 2])


def test_lightning_scan_is_a_decaying_sum():
    r = np.random.default_rng(2)
    q, k, v = r.standard_normal((2, 5, 3)), r.standard_normal((2, 5, 3)), r.standard_normal((2, 5, 4))
    d = np.array([0.5, 1.0])
    o = L.lightning_scan(q, k, v, d)
    want = sum(d[:, None] ** (4 - j) * np.einsum("hd,hd->h", q[:, 4], k[:, j])[:, None] * v[:, j] for j in range(5))
    assert np.allclose(o[:, 4], want)


def test_delta_scan_replaces_what_a_key_held():
    """No decay and full removal: writing twice under one unit key leaves the second value; another key's value stays."""
    e = np.eye(3)
    one = np.ones((1, 3, 3))
    k = np.stack([e[0], e[1], e[0]])[None]
    v = np.array([[[1.0, 2, 3], [4, 5, 6], [7, 8, 9]]])
    r = np.stack([e[0], e[0], e[0] + e[1]])[None]
    o = L.delta_scan(r, k, v, one, one)
    assert np.allclose(o[0], [[1, 2, 3], [1, 2, 3], [11, 13, 15]], atol=1e-5)


def test_decay_bounds_and_unit_key():
    W = {"w1": np.zeros((1, 2)), "w2": np.zeros((3, 1)), "w0": np.array([-50.0, 0.0, 50.0])}
    assert np.allclose(L.channel_decay(np.zeros((1, 2)), W, "")[0], [1.0, np.exp(-0.5 * np.exp(-0.5)), np.exp(-np.exp(-0.5))])
    assert np.allclose(L.unit_key(np.array([3e-3, 4e-3])), np.array([3e-3, 4e-3]) / np.sqrt(25e-6 + 1e-6))
    assert np.array_equal(L.squared_relu(np.array([-2.0, 3.0])), [0.0, 9.0])


def test_last_position_does_not_depend_on_later_tokens():
    cfg = M.varied()
    W = M.weights(cfg)
    ids = M.tokens(cfg, 40)
    assert np.allclose(L.forward(cfg, W, ids)[0][:25], L.forward(cfg, W, ids[:25])[0])


# ── the GPU tests' inputs expose mistakes ───────────────────────────────────
def changed(cfg, W, ids, patch):
    want, _ = L.forward(cfg, W, ids)
    old = {k: getattr(L, k) for k in patch}
    try:
        for k, f in patch.items():
            setattr(L, k, f)
        return M.error(L.forward(cfg, W, ids)[0], want)
    finally:
        for k, f in old.items():
            setattr(L, k, f)


def test_planted_mistakes_show():
    cfg = M.varied()
    W = M.weights(cfg, seed=2, sharp=2.0)
    ids = M.tokens(cfg, 90)
    mask, rot, delta, decay, light = L.window_mask, L.rotate_halves, L.delta_scan, L.channel_decay, L.lightning_scan

    def neighbours(x, pos, dims, base):
        out = np.array(x)
        a = L.angles(pos, dims, base)
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
        return out

    def lost(f, at):                                          # a state that starts again at a token
        return lambda *x: np.concatenate([f(*[y[:, :at] if np.ndim(y) > 1 else y for y in x]), f(*[y[:, at:] if np.ndim(y) > 1 else y for y in x])], 1)

    for name, patch in {
        "window one wider": dict(window_mask=lambda T, s: mask(T, s + 1)),
        "window one narrower": dict(window_mask=lambda T, s: mask(T, max(1, s - 1))),
        "neighbouring pairs": dict(rotate_halves=neighbours),
        "positions one off late": dict(rotate_halves=lambda x, p, d, b: rot(x, np.where(np.abs(p) > 60, p + 1, p), d, b)),
        "values not rotated": dict(rotated_values=lambda v, p, b: v),
        "mixture not turned back": dict(turned_back=lambda o, p, b: o),
        "removal reads the decayed state": dict(delta_scan=lambda r, k, v, w, a: delta(r, k, v, w, a * w)),
        "removal not by the unit key": dict(unit_key=lambda k: k),
        "no removal": dict(removal_rate=lambda h, W, p: np.zeros((h.shape[0], W[p + "a.b"].size))),
        "no channel decay": dict(channel_decay=lambda h, W, p: np.ones((h.shape[0], W[p + "w0"].size))),
        "decay without its factor": dict(channel_decay=lambda h, W, p: decay(h, W, p) ** np.exp(0.5)),
        "delta state lost": dict(delta_scan=lost(delta, 70)),
        "lightning state lost": dict(lightning_scan=lost(light, 70)),
        "no silu": dict(silu=lambda z: z),
        "relu not squared": dict(squared_relu=lambda z: np.maximum(z, 0)),
        "no cap": dict(output_logits=lambda x, W, c: (L.rms(x, c["norm"]["eps"]) * W["final.norm"]) @ W["embed"].T * c["logit_scale"]),
        "no gates": dict(sigmoid=lambda z: np.ones_like(z), silu=L.silu),
    }.items():
        e = changed(cfg, W, ids, patch)
        assert np.max(e) > 0.05, (name, float(np.max(e)))


@pytest.mark.parametrize("window", [16, 64])
def test_marker_places_are_sharp(window):
    cfg, W = M.marker_attention(window)
    ids = (1 + np.arange(window + 10) % 50).astype(np.uint32)
    ids[4] = M.MARK
    wide = json.loads(json.dumps(cfg))
    wide["layers"][0]["mixer"]["mask"]["size"] = window + 1
    e = M.error(L.forward(wide, W, ids)[0], L.forward(cfg, W, ids)[0])
    assert e[4 + window] > 0.25 and np.all(e[:4 + window] < 1e-9)


@pytest.mark.parametrize("kind", ["lightning", "general_delta"])
def test_marked_states_are_sharp(kind):
    cfg, W = M.marker_state(kind)
    ids = (1 + np.arange(300) % 50).astype(np.uint32)
    with_it = ids.copy()
    with_it[4] = M.MARK
    e = M.error(L.forward(cfg, W, with_it)[0], L.forward(cfg, W, ids)[0])
    assert np.all(e[4:] > 0.25) and np.all(e[:4] < 1e-9)


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
    assert st == _lib.SP_OK and (d.arch, d.n_layers, d.hidden, d.vocab) == (2, 9, 90, 153)
    assert ForwardEngine.arch_block("Tedelix") == 2
    plain = M.varied()
    del plain["logit_softcap"], plain["logit_scale"], plain["layers"][0]["mlp"]
    assert create(plain)[0] == _lib.SP_OK


@pytest.mark.parametrize("path,value,word", [
    (["vocab"], None, "vocab"), (["width"], 0, "width"), (["norm"], None, "norm"), (["layers"], [], "layers"), (["logit_scale"], "x", "logit_scale"),
    (["layers", 1, "type"], "latent_attention", "type"), (["layers", 1, "mixer", "kv_heads"], 4, "kv_heads"), (["layers", 1, "mixer", "rot", "dims"], 22, "rot"),
    (["layers", 1, "mixer", "rot", "dims"], 7, "rot"), (["layers", 1, "mixer", "rot", "base"], None, "base"), (["layers", 1, "mixer", "vdim"], 9, "vdim"),
    (["layers", 1, "mixer", "mask", "size"], 0, "size"), (["layers", 1, "mixer", "scale"], None, "scale"), (["layers", 2, "mixer", "decay"], [0.5], "decay"),
    (["layers", 2, "mixer", "decay"], None, "decay"), (["layers", 2, "mixer", "decay"], [0.1, 0.2, 0.3, 0.4, "x"], "decay"), (["layers", 0, "mixer", "dim"], 1000, "dim"),
    (["layers", 0, "mixer", "heads"], 1.5, "heads"), (["layers", 0, "mlp", "kind"], "moe", "kind"), (["layers", 0, "mlp", "ff"], None, "ff")])
def test_bad_configurations_are_named(path, value, word):
    cfg = M.varied()
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
    cfg = synth.tedelix_config(layers=["general_delta", "attention", "lightning"], width=48, heads=4, kv_heads=2, dim=8, vdim=12, state_heads=3, state_dim=8,
                               state_vdim=12, window=9, ff=20, vocab=30)
    a = {k: tuple(v.shape) for k, v in synth.tedelix_weights(cfg, 0, rank=5).items()}
    for l in cfg["layers"]:
        l["mixer"]["_rank"] = 5
    assert a == {k: tuple(np.shape(v)) for k, v in M.weights(cfg).items()}
