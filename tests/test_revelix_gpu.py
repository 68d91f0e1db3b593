"""Revelix on the CUDA engine against the plain restatement in oracle/revelix.py: float32 engines to 1e-4 of the logits' spread,
bfloat16 ones to a few percent."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import revelix_models as M
from oracle import revelix as L
from sapient_b200._lib import SapientCudaError
from sapient_b200.batching import ContinuousBatcher
from sapient_b200.engine import ForwardEngine

pytestmark = pytest.mark.gpu
TOL = {"float32": 1e-4, "bfloat16": 0.08}
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
mixed_layers = M.mixed_layers


def engine(cfg, W, dtype, **kw):
    kw.setdefault("max_ctx", 512)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_tokens", 512)
    return ForwardEngine.from_config(cfg, W, dtype=dtype, **kw)


def check(got, want, dtype):
    e = M.error(got, want)
    assert np.all(e <= TOL[dtype]), (dtype, float(e.max()), int(np.argmax(e > TOL[dtype])))


def places(n):
    return list(range(n))


def all_logits(eng, ids, slot=0):
    eng.reset_cache(slot)
    return eng.forward_mixed([(slot, ids, places(len(ids)))])


def in_portions(eng, ids, sizes, slot=0):
    eng.reset_cache(slot)
    got, at, k = [], 0, 0
    while at < len(ids):
        part = ids[at:at + sizes[k % len(sizes)]]
        got.append(eng.forward_mixed([(slot, part, places(len(part)))]))
        at += len(part)
        k += 1
    return np.concatenate(got)


# ── each mechanism alone ────────────────────────────────────────────────────
@BOTH
@pytest.mark.parametrize("keep", [["retention"], ["left"], ["right"], ["left", "right"], ["ff"], []], ids=str)
def test_each_mechanism_alone(keep, dtype):
    cfg = M.config([M.retention(ff=44) if keep == ["retention"] else M.parallel()])
    W = M.only(M.weights(cfg, seed=3), *keep)
    ids = M.tokens(cfg, 90)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(all_logits(eng, ids[:7]), want[:7], dtype)
    eng.close()


LEFT = [{"scale": 0.01}, {"scale": 1.5}, {"softcap": 0.5}, {"softcap": 1e4}, {"window": 1}, {"window": 2}, {"window": 16}, {"window": 4000}, {"keep": 0}, {"keep": 1}, {"keep": 16},
        {"keep": 17}, {"keep": 70}, {"window": 1, "keep": 33}, {"window": 16, "keep": 16}, {"base": 3.0}, {"base": 5e5}, {"rot": 0}, {"rot": 2}, {"rot": 20}, {"scaling": None},
        {"scaling": {"factor": 1.0, "original": 10, "fast": 4.0, "slow": 1.0}}, {"scaling": {"factor": 8.0, "original": 3000, "fast": 32.0, "slow": 1.0}, "rot": 20},
        {"scaling": {"factor": 2.5, "original": 100, "fast": 1.0, "slow": 0.9}, "rot": 20}, {"conv": 1}, {"conv": 2}, {"conv": 9}, {"conv": 32}, {"kv_heads": 1}, {"kv_heads": 6},
        {"heads": 1, "kv_heads": 1}, {"heads": 9, "kv_heads": 1}, {"heads": 9, "kv_heads": 9}, {"heads": 20, "kv_heads": 1}, {"heads": 20, "kv_heads": 4}, {"heads": 21, "kv_heads": 7},
        {"heads": 24, "kv_heads": 24}, {"heads": 34, "kv_heads": 2}, {"heads": 40, "kv_heads": 5}, {"heads": 96, "kv_heads": 12}, {"dim": 1, "rot": 0}, {"dim": 130}, {"dim": 256, "vdim": 256},
        {"vdim": 1}, {"vdim": 2}, {"vdim": 33}, {"vdim": 70}, {"vdim": 150}, {"dim": 270}, {"vdim": 300}, {"heads": 40, "kv_heads": 20, "dim": 200, "vdim": 200},
        {"heads": 16, "kv_heads": 4, "dim": 64, "vdim": 64}, {"heads": 10, "kv_heads": 1, "dim": 128, "vdim": 128}, {"heads": 24, "kv_heads": 12, "dim": 128, "vdim": 128, "rot": 128},
        {"heads": 40, "kv_heads": 5, "dim": 64, "vdim": 64, "window": 50, "softcap": 90.0}, {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "window": 4000},
        {"heads": 16, "kv_heads": 16, "dim": 128, "vdim": 128}, {"heads": 18, "kv_heads": 6, "dim": 64, "vdim": 64}]


@pytest.mark.parametrize("change", LEFT, ids=lambda c: "-".join(f"{k}{v}" for k, v in c.items()))
def test_attention_sizes_and_constants(change):
    cfg = M.config([M.parallel(M.left(**change), ff=None)], width=60)
    W = M.only(M.weights(cfg, seed=5, sharp=2.0), "left")
    ids = M.tokens(cfg, 100)
    want, _ = L.forward(cfg, W, ids)
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, W, dtype)
        check(all_logits(eng, ids), want, dtype)
        check(in_portions(eng, ids, [9, 50, 1], slot=1), want, dtype)
        eng.close()


STATES = [("right", dict(heads=h, dim=d, vdim=v)) for h, d, v in ((1, 1, 1), (2, 16, 3), (4, 33, 50), (3, 64, 64), (2, 100, 20), (2, 128, 128), (1, 150, 40), (1, 290, 16), (17, 6, 7), (2, 50, 300))]
STATES += [("retention", dict(heads=h, dim=d, vdim=v, rot=r)) for h, d, v, r in ((1, 1, 1, 0), (8, 16, 64, 16), (9, 40, 17, 2), (33, 8, 4, 8), (2, 128, 128, 128), (2, 50, 300, 50), (1, 260, 30, 100),
                                                                             (3, 33, 20, 32))]
STATES += [("retention", dict(heads=3, decay=[0.0, 1.0, 0.5], base=2.0)), ("retention", dict(heads=2, base=1e6, rot=24))]


@pytest.mark.parametrize("kind,sizes", STATES, ids=str)
def test_state_sizes_and_constants(kind, sizes):
    cfg = M.config([M.retention(**sizes) if kind == "retention" else M.parallel(b=M.right(**sizes), ff=None)], width=60)
    W = M.only(M.weights(cfg, seed=6), kind)
    ids = M.tokens(cfg, 75)
    want, _ = L.forward(cfg, W, ids)
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, W, dtype)
        check(all_logits(eng, ids), want, dtype)                        # scan
        check(in_portions(eng, ids, [40, 3, 1, 31], slot=1), want, dtype)  # scan, then steps of several rows, then a row
        eng.close()


@BOTH
def test_gates_that_forget_everything_or_nothing(dtype):
    """Channels whose gate is next to zero for some tokens, next to one for others: products of decays leave the range of floats."""
    cfg = M.config([M.parallel(b=M.right(heads=2, dim=24, vdim=20), ff=None)], width=64)
    W = M.only(M.weights(cfg, seed=7), "right")
    W["l0.mix.right.lower"][:] = 0.0
    W["l0.mix.right.f"] = M.bf16(W["l0.mix.right.f"] * 12)
    ids = M.tokens(cfg, 200)
    f = L.forget(L.tanh_norm(W["embed"][ids], W, "l0.norm1").astype(np.float64), W, "l0.mix.right.")
    assert f.min() < 1e-12 and (1 - f).min() < 1e-12
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(in_portions(eng, ids, [35, 1, 2], slot=1), want, dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("change", [dict(scale=1.0), dict(scale=None), dict(scale=2.5), dict(eps=0.3)], ids=str)
def test_constants_of_the_stream_and_layers_out(change, dtype):
    """The stream after every layer; eps large enough to matter."""
    cfg = M.config(M.varied()["layers"], vocab=90, width=76, **change)
    ref = {**cfg, "logit_scale": cfg["logit_scale"] or 1.0}
    if cfg["logit_scale"] is None:
        del cfg["logit_scale"]
    W = M.weights(cfg, seed=8)
    ids = M.tokens(cfg, 40)
    want, stream = L.forward(ref, W, ids)
    eng = engine(cfg, W, dtype)
    eng.set_trace(True)
    check(all_logits(eng, ids), want, dtype)
    for i in range(len(cfg["layers"])):
        assert np.max(np.abs(eng.layer_out(i) - stream[i])) < TOL[dtype] * np.std(stream[i]) * 2, i
    eng.close()


@BOTH
def test_what_a_configuration_may_leave_out(dtype):
    """No window, kept keys, cap, convolution, scales: as values that change nothing."""
    cfg = M.config([M.parallel(M.left(window=10 ** 6, keep=0, conv=1, softcap=1e6, scaling=None), left_scale=1.0, right_scale=1.0)])
    W = M.weights(cfg, seed=10)
    for n in ("q", "k", "v"):
        W[f"l0.mix.left.{n}.conv"][:] = 1.0
    ids = M.tokens(cfg, 80)
    want, _ = L.forward(cfg, W, ids)
    m = cfg["layers"][0]["mixer"]
    del m["left_scale"], m["right_scale"], m["left"]["mask"], m["left"]["softcap"], m["left"]["conv"]
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(in_portions(eng, ids, [33, 1, 2], slot=1), want, dtype)
    eng.close()


@BOTH
def test_activation_far_from_zero(dtype):
    cfg = M.config([M.retention(ff=61)], width=64)
    W = M.only(M.weights(cfg, seed=9), "ff")
    W["l0.mlp.up"] = M.bf16(W["l0.mlp.up"] * 6)
    W["l0.mlp.act"][:] = [-3.0, 2.0]
    ids = M.tokens(cfg, 50)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(all_logits(eng, ids[:9]), want[:9], dtype)
    eng.close()


# ── whole prompts, decoding, portions, batches ──────────────────────────────
@BOTH
def test_varied_layers_prompt_and_decode(dtype):
    cfg = M.varied()
    W = M.weights(cfg, seed=4)
    ids = M.tokens(cfg, 150)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(in_portions(eng, ids[:100], [1]), want[:100], dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("sizes", [[2], [3, 1], [15, 16, 17], [31, 2, 33], [40], [64, 5], [100, 1, 1]], ids=str)
def test_portions_of_any_size(sizes, dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=2, sharp=2.0)
    ids = M.tokens(cfg, 150)
    eng = engine(cfg, W, dtype)
    check(in_portions(eng, ids, sizes, slot=2), L.forward(cfg, W, ids)[0], dtype)
    eng.close()


@BOTH
def test_prompt_longer_than_a_chunk_of_the_engine(dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=2)
    ids = M.tokens(cfg, 150)
    want, _ = L.forward(cfg, W, ids)
    for rows in (1, 20, 37, 64):
        eng = engine(cfg, W, dtype, max_tokens=rows)
        check(all_logits(eng, ids), want, dtype)
        eng.close()


@BOTH
def test_mixed_batches_equal_each_request_alone(dtype):
    """Portions beside single tokens, requests left out of a step, slots, states and pages handed on; the pool holds no page
    more than the live requests need."""
    cfg = mixed_layers()
    W = M.weights(cfg, seed=4, sharp=2.0)
    lens = [120, 5, 77, 33, 60, 18, 1, 50]
    reqs = {r: M.tokens(cfg, n, seed=r) for r, n in enumerate(lens)}
    want = {r: L.forward(cfg, W, t)[0] for r, t in reqs.items()}
    eng = engine(cfg, W, dtype, kv_pages=sum(sorted(-(-n // 16) for n in lens)[-4:]))
    at = {r: 0 for r in reqs}
    slot, free, waiting = {}, [3, 2, 1, 0], list(reqs)
    rng = np.random.default_rng(7)
    steps = 0
    while any(at[r] < len(reqs[r]) for r in reqs):
        while waiting and free:
            slot[waiting[0]] = free.pop()
            waiting.pop(0)
        entries, expect = [], []
        for r in list(slot):
            if rng.random() < 0.25:
                continue
            n = min(len(reqs[r]) - at[r], int(rng.choice([1, 1, 2, 7, 40])))
            w = sorted(rng.choice(n, size=int(rng.integers(0, n + 1)), replace=False).tolist())
            entries.append((slot[r], reqs[r][at[r]:at[r] + n], w))
            expect += [want[r][at[r] + i] for i in w]
            at[r] += n
        if not entries:
            continue
        got = eng.forward_mixed(entries)
        steps += 1
        if expect:
            check(got, np.stack(expect), dtype)
        for r in list(slot):
            if at[r] == len(reqs[r]):
                eng.reset_cache(slot[r])
                free.append(slot.pop(r))
    assert steps > 8
    eng.close()


@BOTH
@pytest.mark.parametrize("n", [12, 80])
def test_rows_of_one_sequence_need_not_stand_together(n, dtype):
    """Tokens of three sequences in turn, as a step of few rows and as one of many, after a prefix in each."""
    cfg = mixed_layers()
    W = M.weights(cfg, seed=5)
    ids = [M.tokens(cfg, 10 + n, seed=s) for s in range(3)]
    want = [L.forward(cfg, W, t)[0] for t in ids]
    eng = engine(cfg, W, dtype)
    for s in (1, 2):                                                    # the sequence of slot 0 starts in the mixed step
        eng.forward_mixed([(s, ids[s][:10], [])])
    rows = [(i, s) for i in range(n // 3) for s in (0, 1, 2, 2)][:32 if n < 32 else None]
    at, entries, expect = [0, 10, 10], [], []
    for _, s in rows:
        entries.append((s, ids[s][at[s]:at[s] + 1], [0]))
        expect.append(want[s][at[s]])
        at[s] += 1
    check(eng.forward_mixed(entries), np.stack(expect), dtype)
    for s in range(3):
        check(eng.forward_mixed([(s, ids[s][at[s]:at[s] + 1], [0])]), want[s][at[s]:at[s] + 1], dtype)
    eng.close()


@BOTH
def test_freed_slots_and_pages_leave_nothing_behind(dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=9, sharp=3.0)
    eng = engine(cfg, W, dtype, max_batch=2, kv_pages=12)
    for seed, n in ((1, 180), (2, 3), (3, 1), (4, 50), (5, 16), (6, 17)):
        ids = M.tokens(cfg, n, seed)
        check(all_logits(eng, ids, slot=seed % 2), L.forward(cfg, W, ids)[0], dtype)
        eng.reset_cache(seed % 2)
    eng.close()


@BOTH
def test_first_tokens_and_long_decoding(dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=12, sharp=2.0)
    ids = M.tokens(cfg, 260)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    for n in (1, 2, 3):
        check(all_logits(eng, ids[:n]), want[:n], dtype)
    check(in_portions(eng, ids, [1]), want, dtype)
    eng.close()


@BOTH
def test_real_sized_layers(dtype):
    """Heads of the sizes that models have, keys split over blocks, long scans."""
    cfg = M.config([M.parallel(M.left(heads=8, kv_heads=2, dim=128, vdim=128, rot=64, window=300, keep=4, conv=4, softcap=30.0), M.right(heads=3, dim=64, vdim=64), ff=300),
                    M.retention(heads=4, dim=128, vdim=96, rot=128, base=1e4),
                    M.parallel(M.left(heads=24, kv_heads=3, dim=64, vdim=96, rot=64, window=1000, keep=20), M.right(heads=2, dim=128, vdim=128), ff=130)], width=264)
    W = M.weights(cfg, seed=13, sharp=2.0)
    ids = M.tokens(cfg, 630)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype, max_ctx=700, max_tokens=700)
    check(all_logits(eng, ids), want, dtype)
    eng.reset_cache(0)
    eng.forward_mixed([(0, ids[:600], [])])
    for a, b in ((600, 602), (602, 619), (619, 620), (620, 630)):
        check(eng.forward_mixed([(0, ids[a:b], places(b - a))]), want[a:b], dtype)
    eng.close()


# ── one token that stands out ───────────────────────────────────────────────
def with_mask(cfg, key, more):
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["left"]["mask"][key] += more
    return other


def prompts_and_decoding(eng, ids, want, inside, outside, dtype):
    check(all_logits(eng, ids)[[inside, outside]], want[[inside, outside]], dtype)
    eng.reset_cache(1)
    eng.reset_cache(2)
    if inside:
        eng.forward_mixed([(1, ids[:inside], []), (2, ids[:inside], [])])
    for p in range(inside, outside + 1):                 # decoded alone
        check(eng.forward_mixed([(1, ids[p:p + 1], [0])]), want[p:p + 1], dtype)
    check(eng.forward_mixed([(2, ids[inside:outside + 1], [0, outside - inside])]), want[[inside, outside]], dtype)  # in one portion


@BOTH
@pytest.mark.parametrize("window", [1, 16, 33, 64, 100])
def test_a_key_just_inside_and_just_outside_the_window(window, dtype):
    cfg, W = M.marker_attention(window, 0)
    eng = engine(cfg, W, dtype)
    for at in (0, 1, 15, 16, 47):                        # first token, page borders
        n = at + window + 3
        ids = (1 + M.tokens(cfg, n, at) % 100).astype(np.uint32)
        ids[at] = M.MARK
        want, _ = L.forward(cfg, W, ids)
        inside, outside = at + window - 1, at + window   # the last query that sees the marker, the first that does not
        moved = M.error(L.forward(with_mask(cfg, "size", 1), W, ids)[0][outside:outside + 1], want[outside:outside + 1])[0]
        assert moved > 3 * TOL[dtype], moved
        prompts_and_decoding(eng, ids, want, inside, outside, dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("keep", [1, 4, 15, 16, 17, 40])
def test_the_last_kept_key_and_the_one_behind_it(keep, dtype):
    """Far behind the window the last kept key is seen and the next one is not, wherever the two stand in their page."""
    window = 21
    cfg, W = M.marker_attention(window, keep)
    eng = engine(cfg, W, dtype)
    for at, seen in ((keep - 1, True), (keep, False)):
        for far in (0, 1, 40, 200):
            inside, outside = at + window - 1 + far, at + window + far
            ids = (1 + M.tokens(cfg, outside + 3, at) % 100).astype(np.uint32)
            ids[at] = M.MARK
            want, _ = L.forward(cfg, W, ids)
            other = L.forward(with_mask(cfg, "keep_first", -1 if seen else 1), W, ids)[0]
            assert M.error(other[outside:outside + 1], want[outside:outside + 1])[0] > 3 * TOL[dtype]
            prompts_and_decoding(eng, ids, want, inside, outside, dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("kind", ["attention", "retention", "forget"])
def test_a_far_token_among_hundreds(kind, dtype):
    """The marker at every kind of place of a long context, found by prompts and by decoded tokens."""
    cfg, W = M.marker_attention(400, 3, heads=12, kv_heads=4) if kind == "attention" else M.marker_state(kind)
    eng = engine(cfg, W, dtype)
    n = 390
    for at in (0, 1, 15, 16, 63, 64, 200, 255, 256, 300, n - 2):
        ids = (1 + M.tokens(cfg, n, at) % 100).astype(np.uint32)
        ids[at] = M.MARK
        want, _ = L.forward(cfg, W, ids)
        gone = ids.copy()
        gone[at] = M.PLAIN
        assert M.error(L.forward(cfg, W, gone)[0][-1:], want[-1:])[0] > 3 * TOL[dtype]
        check(all_logits(eng, ids)[-40:], want[-40:], dtype)
        eng.reset_cache(1)
        eng.forward_mixed([(1, ids[:-1], [])])
        check(eng.forward_mixed([(1, ids[-1:], [0])]), want[-1:], dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("sink", [-30.0, 6.0, 29.0])
def test_sinks_of_any_size(sink, dtype):
    """From one that counts nothing to one above every score."""
    cfg, W = M.marker_attention(50, 2)
    W["l0.mix.left.sink"][:] = sink
    ids = (1 + M.tokens(cfg, 200, 3) % 100).astype(np.uint32)
    ids[[0, 70]] = M.MARK
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(in_portions(eng, ids, [1, 20, 50, 60], slot=1), want, dtype)
    eng.close()


# ── rollback ────────────────────────────────────────────────────────────────
@BOTH
def test_truncation_goes_back_to_a_checkpoint(dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=15)
    ids = M.tokens(cfg, 90)
    want, _ = L.forward(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    eng.forward_mixed([(1, ids[:40], []), (0, ids[:9], [])])
    eng.checkpoint(1)
    eng.forward_mixed([(1, M.tokens(cfg, 30, 5), [])])
    assert eng.truncate_cache(70, slot=1) == 70          # nothing to cut
    assert eng.truncate_cache(55, slot=1) == 40 and eng.seq_len(1) == 40
    check(eng.forward_mixed([(1, ids[40:], places(50))]), want[40:], dtype)
    assert eng.truncate_cache(39, slot=1) == 0           # before the checkpoint: from the start
    check(eng.forward_mixed([(1, ids[:50], places(50))]), want[:50], dtype)
    assert eng.truncate_cache(45, slot=1) == 0           # the checkpoint belonged to the sequence that is gone
    check(eng.forward_mixed([(0, ids[9:20], places(11))]), want[9:20], dtype)  # the other slot has not noticed
    with pytest.raises(SapientCudaError):
        eng.adopt_prefix(2, [eng.slot_page(0, 0)])
    eng.close()


# ── generation through the framework's entry points ─────────────────────────
def oracle_greedy(cfg, W, prompt, n):
    ids, gaps = list(prompt), []
    for _ in range(n):
        z = L.forward(cfg, W, ids)[0][-1]
        top = np.sort(z)[-2:]
        gaps.append(top[1] - top[0])
        ids.append(int(np.flatnonzero(z == z.max())[-1]))
    gaps = np.asarray(gaps)
    return ids[len(prompt):], int(np.argmax(gaps < 1e-3)) if (gaps < 1e-3).any() else n  # up to a near tie


def test_greedy_generation_through_the_scheduler():
    cfg = mixed_layers()
    W = M.lively(cfg, 31)
    prompts = [M.tokens(cfg, n, seed=50 + n) for n in (3, 40, 17, 90, 64)]
    prompts.append(np.concatenate([prompts[4], M.tokens(cfg, 5, 99)]))   # starts like the one before: states are not shared
    eng = engine(cfg, W, "float32", max_batch=3, kv_pages=30)
    b = ContinuousBatcher(eng, prefill_chunk=37)
    rids = [b.submit(p, 12) for p in prompts[:4]]
    for _ in range(6):
        b.step()
    rids.append(b.submit(prompts[4], 12))
    b.run()
    rids.append(b.submit(prompts[5], 12))
    b.run()
    seen = set()
    for rid, p in zip(rids, prompts):
        got, done = b.poll(rid)
        want, upto = oracle_greedy(cfg, W, p, 12)
        assert done and list(got[:upto]) == want[:upto]
        seen |= set(want)
    assert len(seen) > 20                                # the model does not just repeat itself
    assert b.stats().shared_tokens == 0
    b.close()
    first = eng.forward_mixed([(0, prompts[0], [len(prompts[0]) - 1])], want_argmax=True)
    toks = [int(first[0])] + eng.decode_greedy(first, [0], 11)[:, 0].tolist()
    want, upto = oracle_greedy(cfg, W, prompts[0], 12)
    assert toks[:upto] == want[:upto]
    eng.close()


def test_bf16_generation_does_not_depend_on_the_batch_or_on_graphs():
    cfg = mixed_layers()
    W = M.lively(cfg, 31)
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


@pytest.mark.parametrize("same_draft", [True, False])
def test_speculative_loops(same_draft):
    """The loop in the library and the schedules on the host, with a draft that agrees and one that does not: rejected drafts
    send both models' states back."""
    from sapient_b200 import speculative

    cfg = mixed_layers()
    W = M.lively(cfg, 32)
    other = M.config([M.parallel(M.left(heads=2, kv_heads=1, dim=12, vdim=10), M.right(heads=2, dim=12, vdim=8), ff=20)], vocab=cfg["vocab"], width=40)
    p = M.tokens(cfg, 20)
    want, upto = oracle_greedy(cfg, W, p, 20)
    a = engine(cfg, W, "float32", max_batch=1)
    b = engine(cfg, W, "float32", max_batch=1) if same_draft else engine(other, M.lively(other, 33), "float32", max_batch=1)
    toks, st = speculative.generate_greedy_device(a, b, p, 20, k=3)
    assert list(toks[:upto]) == want[:upto] and (st.accepted_drafts > 0) == same_draft
    toks, _ = speculative.generate_greedy(a, b, p, 20, k=3)
    assert list(toks[:upto]) == want[:upto]
    a.reset_cache()
    b.reset_cache()
    toks, _ = speculative.generate(a, b, p, 20, k=3, rand=lambda: 0.5 if same_draft else 1.0)
    if same_draft:
        assert list(toks[:upto]) == want[:upto]
    a.close()
    b.close()


# ── files and programs ──────────────────────────────────────────────────────
def write_dir(path, cfg, W):
    import torch

    from sapient_b200 import synth

    synth.write_safetensors(str(path), cfg, {k: torch.tensor(v).to(torch.bfloat16) for k, v in W.items()})


def test_a_model_directory_and_the_trace_program(tmp_path):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=42)
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
        check(np.fromfile(out / "0.f32", "<f4").reshape(2, -1), want[[49, 3]], dtype)
        check(np.fromfile(out / "2.f32", "<f4").reshape(3, -1), want[[50, 69, 0]], dtype)


def test_generate_command(tmp_path):
    cfg = mixed_layers()
    W = M.lively(cfg, 41)
    write_dir(tmp_path / "m", cfg, W)
    p = M.tokens(cfg, 6).tolist()
    want, upto = oracle_greedy(cfg, W, p, 5)
    cmd = [sys.executable, "-m", "sapient_b200.generate", "--model", str(tmp_path / "m"), "--dtype", "float32", "--prompt", ",".join(map(str, p)), "--prompt", "1,2",
           "--max-new", "5"]
    for extra in ([], ["--temperature", "0.8", "--seed", "3"]):
        r = subprocess.run(cmd + extra, capture_output=True, text=True, timeout=120, cwd=ROOT)
        assert r.returncode == 0, r.stderr[-2000:]
        lines = [json.loads(x) for x in r.stdout.splitlines() if x.startswith("{")]
        assert len(lines) == 2 and len(lines[1]["tokens"]) == 5
        if not extra:
            assert lines[0]["tokens"][:upto] == want[:upto]
