"""Lepalorn on the CUDA engine against the plain restatement in oracle/lepalorn.py.

float32 engines are held to 1e-4 of the logits' spread, bfloat16 ones to a few percent. A bfloat16 run may choose another
expert than the oracle where two router logits almost tie, so bfloat16 models either use every expert (the choice is
then fixed, the weights are not) or are judged on all but a few positions."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import plan_models as M
from oracle import lepalorn as L
from sapient_b200.batching import ContinuousBatcher
from sapient_b200.engine import ForwardEngine

pytestmark = pytest.mark.gpu
TOL = {"float32": 1e-4, "bfloat16": 0.05}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def engine(cfg, W, dtype, **kw):
    kw.setdefault("max_ctx", 512)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_tokens", 512)
    return ForwardEngine.from_config(cfg, W, dtype=dtype, **kw)


def fixed_choice():
    """Two layers whose tokens use every expert; sizes that are no multiples of anything."""
    return M.config([(M.mixer(heads=5, dim=20, rot=10, vdim=28, rank=52, window=37), M.moe(experts=3, top=3, ff=44, shared=(20, 0.7))),
                     (M.mixer(heads=3, dim=33, rot=10, vdim=17, rank=52, window=70, kv_from=0), M.moe(experts=2, top=2, ff=12, shared=None))],
                    vocab=133, width=76)


def check(got, want, dtype, allow=0.0):
    e = M.error(got, want)
    bad = np.mean(e > TOL[dtype])
    assert bad <= allow, (dtype, float(e.max()), float(bad), int(np.argmax(e > TOL[dtype])))


def all_logits(eng, ids, slot=0):
    eng.reset_cache(slot)
    return eng.forward_mixed([(slot, ids, list(range(len(ids))))])


# ── each mechanism alone ────────────────────────────────────────────────────
def isolate(W, cfg, keep):
    """Turns everything off but `keep`: gains of the other sublayers to zero, depth averages to the newest result."""
    W = dict(W)
    for i in range(len(cfg["layers"])):
        p = f"l{i}."
        if keep != "attention":
            W[p + "norm1"] = np.zeros((), np.float32)
        if keep not in ("experts", "shared") and p + "norm2" in W:
            W[p + "norm2"] = np.zeros((), np.float32)
        if keep == "shared":
            W.update({n: np.zeros_like(v) for n, v in W.items() if n.startswith(p + "mlp.e") and n.endswith("down")})
        if keep == "experts":
            W.update({n: np.zeros_like(v) for n, v in W.items() if n.startswith(p + "mlp.shared.down")})
        if keep != "depth":
            W[p + "dwa"] = np.eye(i + 2, dtype=np.float32)[-1]
    return W


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("keep", ["attention", "experts", "shared", "depth", "nothing"])
def test_each_mechanism_alone(keep, dtype):
    cfg = fixed_choice()
    W = isolate(M.weights(cfg, seed=3), cfg, keep)
    ids = M.tokens(cfg, 90)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(all_logits(eng, ids[:7]), want[:7], dtype)
    eng.close()


@pytest.mark.parametrize("change", [{"scale": 0.01}, {"scale": 1.5}, {"window": 1}, {"window": 2}, {"base": 3.0}, {"base": 5e5}, {"rot": 2}, {"rot": 46},
                                    {"heads": 1}, {"heads": 16}, {"heads": 33}, {"rank": 8}, {"rank": 200}, {"vdim": 3}, {"dim": 1}],
                         ids=lambda c: "-".join(f"{k}{v}" for k, v in c.items()))
def test_attention_sizes_and_constants(change):
    cfg = M.config([(M.mixer(**{**dict(heads=4, dim=18, rot=6, vdim=14, rank=30, window=21), **change}), None)], width=60)
    W = M.weights(cfg, seed=5)
    ids = M.tokens(cfg, 70)
    want, _ = L.forward(cfg, W, ids)
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, W, dtype)
        check(all_logits(eng, ids), want, dtype)
        check(np.concatenate([eng.forward_mixed([(1, ids[i:i + 9], list(range(len(ids[i:i + 9]))))]) for i in range(0, 70, 9)]), want, dtype)
        eng.close()


@pytest.mark.parametrize("change", [dict(experts=1, top=1), dict(experts=40, top=1), dict(experts=40, top=7), dict(limit=0.05), dict(limit=50.0),
                                    dict(ff=1), dict(ff=130), dict(shared=None), dict(shared=(200, 0.1))], ids=str)
def test_experts_sizes_and_constants(change):
    cfg = M.config([(M.mixer(), M.moe(**change))], width=72)
    W = isolate(M.weights(cfg, seed=6), cfg, "experts" if change.get("shared", 0) is None else "all")
    W["l0.norm2"] = np.float32(1.0)
    ids = M.tokens(cfg, 80)
    want, _ = L.forward(cfg, W, ids)
    for dtype, allow in (("float32", 0.0), ("bfloat16", 0.08)):
        eng = engine(cfg, W, dtype)
        check(all_logits(eng, ids), want, dtype, allow)
        check(all_logits(eng, ids[:20]), want[:20], dtype, allow)
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_scale_eps_and_layers_out(dtype):
    """eps large enough to matter, and the stream after every layer."""
    cfg = fixed_choice()
    cfg["norm"]["eps"] = 0.3
    cfg["embedding"]["scale"] = 0.11
    W = M.weights(cfg, seed=8)
    ids = M.tokens(cfg, 40)
    want, stream = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    eng.set_trace(True)
    check(all_logits(eng, ids), want, dtype)
    for i in range(len(cfg["layers"])):
        assert np.max(np.abs(eng.layer_out(i) - stream[i])) < TOL[dtype] * np.std(stream[i]) * 2
    eng.close()


# ── whole prompts, decoding, portions, batches ──────────────────────────────
@pytest.mark.parametrize("dtype,allow", [("float32", 0.0), ("bfloat16", 0.15)])
def test_varied_layers_prompt_decode_and_portions(dtype, allow):
    cfg = M.varied()
    W = M.weights(cfg, seed=1)
    ids = M.tokens(cfg, 150)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype, allow)
    eng.reset_cache(0)
    got = [eng.forward_mixed([(0, ids[i:i + 1], [0])]) for i in range(100)]
    check(np.concatenate(got), want[:100], dtype, allow)
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [[2], [3, 1], [15, 16, 17], [31, 2, 33], [40], [64, 5], [100, 1, 1]], ids=str)
def test_portions_of_any_size(sizes, dtype):
    cfg = fixed_choice()
    W = M.weights(cfg, seed=2, sharp=2.0)
    n = 150
    ids = M.tokens(cfg, n)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    got, at, k = [], 0, 0
    while at < n:
        part = ids[at:at + sizes[k % len(sizes)]]
        got.append(eng.forward_mixed([(2, part, list(range(len(part))))]))
        at += len(part)
        k += 1
    check(np.concatenate(got), want, dtype)
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_longer_than_a_chunk_of_the_engine(dtype):
    cfg = fixed_choice()
    W = M.weights(cfg, seed=2)
    ids = M.tokens(cfg, 150)
    want, _ = L.forward(cfg, W, ids)
    for rows in (1, 20, 37, 64):
        eng = engine(cfg, W, dtype, max_tokens=rows)
        check(all_logits(eng, ids), want, dtype)
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_each_request_alone(dtype):
    """Portions beside single tokens, requests left out of a step, slots and pages handed on; the pool holds no page more
    than the live requests need."""
    cfg = fixed_choice()
    W = M.weights(cfg, seed=4, sharp=2.0)
    reqs = {r: M.tokens(cfg, n, seed=r) for r, n in enumerate([120, 5, 77, 33, 60, 18])}
    want = {r: L.forward(cfg, W, t)[0] for r, t in reqs.items()}
    pages = sum(-(-n // 16) for n in (120, 5, 77, 33)) + 2
    eng = engine(cfg, W, dtype, kv_pages=pages)
    at = {r: 0 for r in reqs}
    slot, free, waiting = {}, [3, 2, 1, 0], list(reqs)
    rng = np.random.default_rng(7)
    steps = 0
    while any(at[r] < len(reqs[r]) for r in reqs):
        while waiting and free:
            slot[waiting[0]] = free.pop()
            waiting.pop(0)
        entries, places = [], []
        for r in list(slot):
            if rng.random() < 0.25:
                continue
            left = len(reqs[r]) - at[r]
            n = min(left, int(rng.choice([1, 1, 2, 7, 40])))
            part = reqs[r][at[r]:at[r] + n]
            w = sorted(rng.choice(n, size=int(rng.integers(0, n + 1)), replace=False).tolist())
            entries.append((slot[r], part, w))
            places += [(r, at[r] + i) for i in w]
            at[r] += n
        if not entries:
            continue
        got = eng.forward_mixed(entries)
        steps += 1
        if places:
            check(got, np.stack([want[r][p] for r, p in places]), dtype)
        for r in list(slot):
            if at[r] == len(reqs[r]):
                eng.reset_cache(slot[r])
                free.append(slot.pop(r))
    assert steps > 8
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_freed_pages_leave_nothing_behind(dtype):
    """A slot that held a long sequence serves short ones afterwards; a truncated one goes on differently."""
    cfg = fixed_choice()
    W = M.weights(cfg, seed=9, sharp=3.0)
    eng = engine(cfg, W, dtype, max_batch=2, kv_pages=12)
    for seed, n in ((1, 180), (2, 3), (3, 1), (4, 50), (5, 16), (6, 17)):
        ids = M.tokens(cfg, n, seed)
        check(all_logits(eng, ids, slot=seed % 2), L.forward(cfg, W, ids)[0], dtype)
        if n < 180:
            eng.reset_cache(seed % 2)
        else:
            eng.reset_cache()
    ids = M.tokens(cfg, 60, 10)
    all_logits(eng, ids)
    eng.truncate_cache(35, 0)
    other = np.concatenate([ids[:35], M.tokens(cfg, 20, 11)])
    check(eng.forward_mixed([(0, other[35:], list(range(20)))]), L.forward(cfg, W, other)[0][35:], dtype)
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(dtype):
    cfg = fixed_choice()
    W = M.weights(cfg, seed=12, sharp=2.0)
    ids = M.tokens(cfg, 260)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    for n in (1, 2, 3):
        check(all_logits(eng, ids[:n]), want[:n], dtype)
    eng.reset_cache(0)
    got = [eng.forward_mixed([(0, ids[i:i + 1], [0])]) for i in range(len(ids))]  # over many window lengths and pages
    check(np.concatenate(got), want, dtype)
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [dict(heads=18, dim=100, rot=64, vdim=200, rank=300, window=90), dict(heads=2, dim=128, rot=64, vdim=128, rank=512, window=300),
                                   dict(heads=3, dim=20, rot=20, vdim=300, rank=640, window=50), dict(heads=20, dim=64, rot=32, vdim=64, rank=160, window=400)],
                         ids=["wide-values", "rank-512", "rank-640", "two-head-groups"])
def test_real_sized_heads(shape, dtype):
    cfg = M.config([(M.mixer(**shape), None), (M.mixer(**shape, kv_from=0), M.moe(experts=2, top=2))], width=200)
    W = M.weights(cfg, seed=13, sharp=2.0)
    ids = M.tokens(cfg, 330)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    eng.reset_cache(0)
    eng.forward_mixed([(0, ids[:300], [])])
    for a, b in ((300, 302), (302, 319), (319, 320)):
        check(eng.forward_mixed([(0, ids[a:b], list(range(b - a)))]), want[a:b], dtype)
    eng.close()


# ── one key that stands out ─────────────────────────────────────────────────
MARK, PLAIN = 0, 1


def marker_model(window, n_layers=1):
    """Every query looks for the marker token: its latent is the only one with a large first coordinate, so that a visible
    marker takes all of the attention and an invisible one leaves a broad mixture. Returns (cfg, W)."""
    cfg = M.config([(M.mixer(heads=4, dim=16, rot=8, vdim=24, rank=36, window=window, scale=0.25), None) for _ in range(n_layers)], width=64)
    W = M.weights(cfg, seed=21)
    e = W["embed"]
    e[:, 0] = 0.0
    e[:, 1] = 4.0
    e[MARK, 0] = 60.0
    for i in range(n_layers):
        p = f"l{i}.mix."
        W[p + "dkv"][:, :2] = 0.0
        W[p + "dkv"][0] = 0.0
        W[p + "dkv"][0, 0] = 1.0
        W[p + "dkv.norm"][:] = 1.0
        q = W[p + "q"].reshape(4, 24, -1)
        q[:, 0, :] = 0.0
        q[:, 0, 1] = 8.0
        W[p + "uk"].reshape(4, 16, -1)[:, 0, :] = 0.0
        W[p + "uk"].reshape(4, 16, -1)[:, 0, 0] = 1.0
    return cfg, {k: M.bf16(v) for k, v in W.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [1, 16, 33, 64, 100])
def test_a_key_just_inside_and_just_outside_the_window(window, dtype):
    cfg, W = marker_model(window)
    wide = json.loads(json.dumps(cfg))
    wide["layers"][0]["mixer"]["mask"]["size"] = window + 1
    eng = engine(cfg, W, dtype)
    for at in (0, 1, 15, 16, 47):                        # first token, page borders
        n = at + window + 3
        ids = np.full(n, PLAIN, np.uint32) + (M.tokens(cfg, n, at) % 100).astype(np.uint32)
        ids[at] = MARK
        want, _ = L.forward(cfg, W, ids)
        inside, outside = at + window - 1, at + window   # the last query that sees the marker, the first that does not
        # the places are sharp: a window one token wider moves the outside one far
        moved = M.error(L.forward(wide, W, ids)[0][outside:outside + 1], want[outside:outside + 1])[0]
        assert moved > 5 * TOL[dtype], moved
        check(all_logits(eng, ids)[[inside, outside]], want[[inside, outside]], dtype)
        eng.reset_cache(1)
        if inside:
            eng.forward_mixed([(1, ids[:inside], [])])
        for p in (inside, outside):
            check(eng.forward_mixed([(1, ids[p:p + 1], [0])]), want[p:p + 1], dtype)
        # and with both places in one short portion
        eng.reset_cache(2)
        if inside:
            eng.forward_mixed([(2, ids[:inside], [])])
        check(eng.forward_mixed([(2, ids[inside:inside + 3], [0, 1])]), want[[inside, outside]], dtype)
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_among_hundreds(dtype):
    """The marker at every kind of place of a long context, found by decoded tokens (split keys) and by prompts."""
    cfg, W = marker_model(400)
    eng = engine(cfg, W, dtype)
    n = 390
    for at in (0, 1, 15, 16, 63, 64, 200, 255, 256, 300, n - 2):
        ids = (1 + M.tokens(cfg, n, at) % 100).astype(np.uint32)
        ids[at] = MARK
        want, _ = L.forward(cfg, W, ids)
        gone = ids.copy()
        gone[at] = PLAIN
        assert M.error(L.forward(cfg, W, gone)[0][-1:], want[-1:])[0] > 5 * TOL[dtype]
        check(all_logits(eng, ids)[-40:], want[-40:], dtype)
        eng.reset_cache(1)
        eng.forward_mixed([(1, ids[:-1], [])])
        check(eng.forward_mixed([(1, ids[-1:], [0])]), want[-1:], dtype)
    eng.close()


# ── generation through the framework's entry points ─────────────────────────
def oracle_greedy(cfg, W, prompt, n):
    ids, gaps = list(prompt), []
    for _ in range(n):
        z = L.forward(cfg, W, ids)[0][-1]
        top = np.sort(z)[-2:]
        gaps.append(top[1] - top[0])
        ids.append(int(np.flatnonzero(z == z.max())[-1]))
    return ids[len(prompt):], np.asarray(gaps)


def test_greedy_generation_through_the_scheduler():
    cfg = fixed_choice()
    W = M.weights(cfg, seed=30)
    prompts = [M.tokens(cfg, n, seed=50 + n) for n in (3, 40, 17, 90, 64)]
    prompts.append(np.concatenate([prompts[4], M.tokens(cfg, 5, 99)]))   # shares whole pages with the one before
    eng = engine(cfg, W, "float32", max_batch=3, kv_pages=30)
    b = ContinuousBatcher(eng, prefill_chunk=37)
    rids = [b.submit(p, 12) for p in prompts[:4]]
    for _ in range(6):
        b.step()
    rids.append(b.submit(prompts[4], 12))
    b.run()
    rids.append(b.submit(prompts[5], 12))
    b.run()
    for rid, p in zip(rids, prompts):
        got, done = b.poll(rid)
        want, gaps = oracle_greedy(cfg, W, p, 12)
        upto = int(np.argmax(gaps < 1e-3)) if (gaps < 1e-3).any() else 12  # up to a near tie
        assert done and list(got[:upto]) == want[:upto]
    assert b.stats().shared_tokens > 0
    b.close()
    first = eng.forward_mixed([(0, prompts[0], [len(prompts[0]) - 1])], want_argmax=True)
    toks = eng.decode_greedy(first, [0], 11)[:, 0]
    want, gaps = oracle_greedy(cfg, W, prompts[0], 12)
    if gaps.min() > 1e-3:
        assert [int(first[0])] + toks.tolist() == want
    eng.close()


def test_bf16_generation_does_not_depend_on_the_batch_or_on_graphs():
    cfg = fixed_choice()
    W = M.weights(cfg, seed=31)
    prompts = [M.tokens(cfg, n, seed=n) for n in (5, 48, 90)]
    eng = engine(cfg, W, "bfloat16")
    for i, p in enumerate(prompts):
        eng.forward_mixed([(i, p, [])])
    first = [1, 2, 3]
    together = eng.decode_greedy(first, [0, 1, 2], 40)
    for i, p in enumerate(prompts):
        eng.reset_cache(i)
        eng.set_graphs(i % 2 == 0)
        eng.forward_mixed([(i, p, [])])
        alone = eng.decode_greedy([first[i]], [i], 40)[:, 0]
        ids = np.concatenate([p, [first[i]], alone]).astype(np.uint32)
        z = L.forward(cfg, W, ids[:-1])[0][len(p):]
        for seq in (alone, together[:, i]):              # every pick is a maximum within the tolerance, up to where the two part
            same = int(np.argmax(seq != alone)) if (seq != alone).any() else 40
            picked = z[np.arange(same), seq[:same].astype(int)]
            assert np.all(z[:same].max(-1) - picked < 6 * TOL["bfloat16"] * z.std())
            assert same >= 10 or z[same].max() - z[same][int(seq[same])] < 6 * TOL["bfloat16"] * z.std()
    eng.close()


def test_speculative_loop_on_a_plan_model():
    from sapient_b200 import speculative

    cfg = fixed_choice()
    W = M.weights(cfg, seed=32)
    p = M.tokens(cfg, 20)
    a, b = engine(cfg, W, "float32", max_batch=1), engine(cfg, W, "float32", max_batch=1)
    toks, st = speculative.generate_greedy_device(a, b, p, 20, k=3)
    want, gaps = oracle_greedy(cfg, W, p, 20)
    if gaps.min() > 1e-3:
        assert list(toks) == want and st.accepted_drafts > 0
    a.close()
    b.close()


# ── files and programs ──────────────────────────────────────────────────────
def write_dir(path, cfg, W):
    import torch

    from sapient_b200 import synth

    synth.write_safetensors(str(path), cfg, {k: torch.tensor(v).to(torch.bfloat16) for k, v in W.items()})


def test_a_model_directory_and_the_trace_program(tmp_path):
    cfg = fixed_choice()
    W = M.weights(cfg, seed=40)
    write_dir(tmp_path / "m", cfg, W)
    ids = M.tokens(cfg, 70)
    want, _ = L.forward(cfg, W, ids)
    eng = ForwardEngine.from_pretrained(str(tmp_path / "m"), dtype="float32", max_ctx=128)
    check(all_logits(eng, ids), want, "float32")
    eng.close()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:50].tolist(), "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": ids[:9].tolist(), "want": []}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[50:].tolist(), "want": [0, 19]}, {"id": "z", "tokens": [int(ids[0])], "want": [0]}], "end": ["x", "z"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=120)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert not (out / "1.f32").exists()
        check(np.fromfile(out / "0.f32", "<f4").reshape(2, -1), want[[49, 3]], dtype)
        check(np.fromfile(out / "2.f32", "<f4").reshape(3, -1), want[[50, 69, 0]], dtype)


def test_generate_command(tmp_path):
    cfg = fixed_choice()
    W = M.weights(cfg, seed=41)
    write_dir(tmp_path / "m", cfg, W)
    p = M.tokens(cfg, 6).tolist()
    want, gaps = oracle_greedy(cfg, W, p, 5)
    r = subprocess.run([sys.executable, "-m", "sapient_b200.generate", "--model", str(tmp_path / "m"), "--dtype", "float32", "--prompt", ",".join(map(str, p)),
                        "--prompt", "1,2", "--max-new", "5"], capture_output=True, text=True, timeout=120, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(x) for x in r.stdout.splitlines() if x.startswith("{")]
    assert len(lines) == 2 and len(lines[1]["tokens"]) == 5
    if gaps.min() > 1e-3:
        assert lines[0]["tokens"] == want
