"""CPU side of the Lepalorn tests: the restatement's mechanisms against hand-made cases, planted mistakes that the GPU
tests' inputs must expose, and the configuration and file readers of the library."""
import ctypes as C
import json
import struct

import numpy as np
import pytest

import plan_models as M
from oracle import lepalorn as L
from sapient_b200 import _lib, synth
from sapient_b200.engine import ForwardEngine
from test_lepalorn_gpu import MARK, fixed_choice, marker_model


# ── the restatement ─────────────────────────────────────────────────────────
def test_rotation_pairs_neighbours_and_keeps_dot_products_relative():
    x = np.zeros((1, 4))
    x[0, 2] = 1.0
    y = L.rotate_interleaved(x, np.array([3]), 100.0)
    assert np.allclose(y[0], [0, 0, np.cos(0.3), np.sin(0.3)])          # 3 * 100^(-2/4) = 0.3
    r = np.random.default_rng(0)
    q, k = r.standard_normal(8), r.standard_normal(8)
    dot = lambda i, j: float(L.rotate_interleaved(q[None], np.array([i]), 50.0)[0] @ L.rotate_interleaved(k[None], np.array([j]), 50.0)[0])  # noqa: E731
    assert abs(dot(9, 4) - dot(105, 100)) < 1e-12 and abs(dot(9, 4) - dot(9, 5)) > 1e-3


def test_window_counts_the_token_itself():
    m = L.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 5
    assert np.array_equal(L.window_mask(4, 1), np.eye(4, dtype=bool))


def test_norms_and_unit():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(L.scalar_rms_norm(x, np.float32(2.0), 0.5), 2 * x / np.sqrt(13.0))
    h, W = np.array([[1.0]]), {"gate": np.array([[5.0]]), "up": np.array([[-7.0]]), "down": np.array([[1.0]])}
    assert np.allclose(L.clamped_expert(h, W, "", 2.0), 2 / (1 + np.exp(-3.404)) * (-2 + 1))  # gate capped above, up both ways
    W["gate"] = np.array([[-5.0]])
    assert np.allclose(L.clamped_expert(h, W, "", 2.0), -5 / (1 + np.exp(8.51)) * (-1))       # the gate has no lower bound


def test_route_softmax_is_over_the_chosen():
    W = {"router": np.eye(4), "router.b": np.array([0.0, 5.0, 0.0, 0.0])}
    pick, w = L.route(np.array([[1.0, 0.0, 3.0, 2.0]]), W, "", 2)
    assert pick.tolist() == [[1, 2]] and np.allclose(w, L.softmax(np.array([[5.0, 3.0]])))


def test_last_position_does_not_depend_on_later_tokens():
    cfg = M.varied()
    W = M.weights(cfg)
    ids = M.tokens(cfg, 40)
    assert np.allclose(L.forward(cfg, W, ids)[0][:25], L.forward(cfg, W, ids[:25])[0])


# ── the GPU tests' inputs expose mistakes ───────────────────────────────────
def changed(cfg, W, ids, **patch):
    """The logits' error when functions of the restatement are replaced."""
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
    cfg = fixed_choice()
    W = M.weights(cfg, seed=2, sharp=2.0)
    ids = M.tokens(cfg, 150)
    mask, rot, sig = L.window_mask, L.rotate_interleaved, L.sigmoid
    halves = lambda x, p, b: np.concatenate([x[..., :x.shape[-1] // 2], x[..., x.shape[-1] // 2:]], -1)  # noqa: E731
    cases = {
        "window one wider": dict(window_mask=lambda T, s: mask(T, s + 1)),
        "window one narrower": dict(window_mask=lambda T, s: mask(T, s - 1)),
        "positions one off on long prompts only": dict(rotate_interleaved=lambda x, p, b: rot(x, np.where(p > 60, p + 1, p), b)),
        "no rotation": dict(rotate_interleaved=halves),
        "no eps": dict(rms_normalise=lambda x, e: x / np.sqrt(np.mean(x * x, -1, keepdims=True))),
        "no gate": dict(sigmoid=lambda z: np.ones_like(z)),
        "depth average dropped": dict(depth_average=lambda h, c: h[-1]),
        "oldest result missing": dict(depth_average=lambda h, c: sum(a * X for a, X in list(zip(c, h))[1:])),
    }
    for name, patch in cases.items():
        e = changed(cfg, W, ids, **patch)
        floor = 1e-4 if name == "no eps" else 0.05
        assert np.max(e) > (2e-7 if name == "no eps" else floor), (name, float(np.max(e)))
    assert sig(0.0) == 0.5


@pytest.mark.parametrize("window", [16, 64])
def test_marker_places_are_sharp(window):
    cfg, W = marker_model(window)
    ids = (1 + np.arange(window + 10) % 50).astype(np.uint32)
    ids[4] = MARK
    wide = json.loads(json.dumps(cfg))
    wide["layers"][0]["mixer"]["mask"]["size"] = window + 1
    e = M.error(L.forward(wide, W, ids)[0], L.forward(cfg, W, ids)[0])
    assert e[4 + window] > 0.25 and np.all(e[:4 + window] < 1e-9)


# ── readers ─────────────────────────────────────────────────────────────────
def create(cfg, ctx=64):
    h, d = C.c_void_p(), ForwardEngine._run_desc(0, ctx, 1, 16, 0)
    text = cfg if isinstance(cfg, bytes) else json.dumps(cfg).encode()
    st = _lib.lib().sp_cuda_engine_create_from_config(text, 30, C.byref(d), C.byref(h))
    if st == _lib.SP_OK:
        out = _lib.SpModelDesc()
        assert _lib.lib().sp_cuda_engine_desc(h, C.byref(out)) == _lib.SP_OK
        _lib.lib().sp_cuda_engine_destroy(h)
        return st, out
    return st, _lib.lib().sp_cuda_last_error().decode()


def test_configuration_is_read_from_the_file():
    st, d = create(M.varied())
    assert st == _lib.SP_OK and (d.arch, d.n_layers, d.hidden, d.vocab) == (2, 6, 90, 151)
    assert ForwardEngine.arch_block("Lepalorn") == 2 and ForwardEngine.arch_block("qwen2") == 0 and ForwardEngine.arch_block("phi2") == 1
    with pytest.raises(_lib.SapientCudaError):
        ForwardEngine.arch_block("nosuch")


def edit(path, value):
    cfg = M.varied()
    at = cfg
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path,value,word", [
    (["vocab"], None, "vocab"), (["width"], 0, "width"), (["norm"], None, "norm"), (["layers"], [], "layers"),
    (["layers", 1, "type"], "conv", "type"), (["layers", 2, "mixer", "kv_from"], 2, "kv_from"), (["layers", 2, "mixer", "kv_from"], 1, "kv_from"),
    (["layers", 3, "mixer", "kv_from"], 2, "kv_from"), (["layers", 0, "mixer", "rot_dim"], 7, "rot"), (["layers", 0, "mixer", "heads"], 1.5, "heads"),
    (["layers", 0, "mlp", "kind"], "dense", "kind"), (["layers", 0, "mlp", "router", "top"], 6, "top"), (["layers", 0, "mlp", "expert", "limit"], None, "limit"),
    (["layers", 0, "mixer", "mask", "size"], 0, "size"), (["layers", 0, "mixer", "scale"], "x", "scale")])
def test_bad_configurations_are_named(path, value, word):
    st, msg = create(edit(path, value))
    assert st == _lib.SP_ERR_ARG and word in msg, msg


def test_other_texts_are_refused():
    assert create(b"{")[0] == _lib.SP_ERR_IO and create(b"[1]")[0] == _lib.SP_ERR_IO
    assert create({"architecture": "gpt2"})[0] == _lib.SP_ERR_DTYPE and create({})[0] == _lib.SP_ERR_ARG
    assert create(M.varied(), ctx=0)[0] == _lib.SP_ERR_ARG


def test_safetensors_headers_are_checked(tmp_path):
    cfg = M.uniform(1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    run = ForwardEngine._run_desc(0, 64, 1, 16, 0)

    def load(head, data=b"\0" * 64, raw=None):
        h = C.c_void_p()
        t = raw if raw is not None else json.dumps(head).encode()
        (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", len(t)) + t + data)
        return _lib.lib().sp_cuda_engine_from_dir(str(tmp_path).encode(), 30, C.byref(run), C.byref(h))

    bad_io, bad_shape = _lib.SP_ERR_IO, _lib.SP_ERR_SHAPE
    one = {"dtype": "BF16", "shape": [4, 8], "data_offsets": [0, 64]}
    assert load({"embed": {**one, "data_offsets": [0, 128]}}) == bad_io
    assert load({"embed": {**one, "data_offsets": [-2, 62]}}) == bad_io
    assert load({"embed": {**one, "data_offsets": [64, 0]}}) == bad_io
    assert load({"embed": {**one, "shape": [4, 9]}}) == bad_shape
    assert load({"embed": {**one, "shape": [-4, -8]}}) == bad_shape
    assert load({"embed": {**one, "shape": [1e300, 1e300]}}) == bad_shape
    assert load({"embed": {**one, "dtype": "I8"}}) == _lib.SP_ERR_DTYPE
    assert load({"embed": {"dtype": "BF16"}}) == bad_io
    assert load({}, raw=b"{not json") == bad_io
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", 1 << 60) + b"{}")
    h = C.c_void_p()
    assert _lib.lib().sp_cuda_engine_from_dir(str(tmp_path).encode(), 30, C.byref(run), C.byref(h)) == bad_io
    assert _lib.lib().sp_cuda_engine_from_dir(str(tmp_path / "none").encode(), 30, C.byref(run), C.byref(h)) == bad_io
    assert _lib.lib().sp_cuda_engine_from_dir(str(tmp_path).encode(), 12, C.byref(run), C.byref(h)) == _lib.SP_ERR_DTYPE


def test_synthetic_builder_makes_the_same_tensors_as_the_tests():
    cfg = synth.lepalorn_config(layers=3, width=48, heads=2, dim=8, rot=4, vdim=8, rank=16, window=9, experts=3, top=2, ff=10, shared_ff=6, vocab=30,
                                shared_latent_from=1)
    a = {k: tuple(v.shape) for k, v in synth.lepalorn_weights(cfg, 0).items()}
    b = {k: tuple(np.shape(v)) for k, v in M.weights(cfg).items()}
    assert a == b
