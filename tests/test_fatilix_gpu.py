"""Fatilix on the CUDA engine against the plain restatement in oracle/fatilix.py: float32 engines to 1e-4 of the logits' spread,
bfloat16 ones to a few percent. A bfloat16 run may choose another expert than the oracle where two choice scores almost tie, so
bfloat16 models either use every expert (the choice is then fixed, the weights are not) or are judged on all but a few
positions."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import fatilix_models as M
from oracle import fatilix as L
from sapient_b200.batching import ContinuousBatcher
from sapient_b200.engine import ForwardEngine

pytestmark = pytest.mark.gpu
TOL = {"float32": 1e-4, "bfloat16": 0.06}
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def engine(cfg, W, dtype, **kw):
    kw.setdefault("max_ctx", 512)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_tokens", 512)
    return ForwardEngine.from_config(cfg, W, dtype=dtype, **kw)


def oracle(cfg, W, ids):
    return L.forward(M.spelled(cfg), W, ids)[0]


def mixed_layers():
    """Both kinds of attention and of feed-forward, every expert chosen; sizes that are no multiples of anything."""
    return M.config([M.biased(heads=6, kv_heads=3, dim=18, vdim=26, bias_max=70, rows=11, mlp=M.dense(30)),
                     M.shared_kv(heads=10, kv_heads=2, dim=22, mlp=M.moe(experts=4, top=4, groups=(2, 2), ff=27, shared=19)),
                     M.biased(heads=3, kv_heads=1, dim=30, vdim=9, bias_max=300, rows=26, mlp=M.moe(experts=3, top=3, groups=None, ff=14, shared=None))],
                    vocab=133, width=76)


def check(got, want, dtype, allow=0.0):
    e = M.error(got, want)
    bad = np.mean(e > TOL[dtype])
    assert bad <= (allow if dtype == "bfloat16" else 0.0), (dtype, float(e.max()), float(bad), int(np.argmax(e > TOL[dtype])))


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
@pytest.mark.parametrize("keep", ["mixer", "ff", "neither"])
@pytest.mark.parametrize("make", ["shared_dense", "shared_moe", "biased_dense", "biased_moe"])
def test_each_sublayer_alone(make, keep, dtype):
    attn, ff = make.split("_")
    mlp = M.dense() if ff == "dense" else M.moe(experts=5, top=5, groups=None)
    cfg = M.config([(M.shared_kv if attn == "shared" else M.biased)(mlp=mlp)])
    W = M.silent(M.weights(cfg, seed=3), *{"mixer": ["l0.norm2"], "ff": ["l0.norm1"], "neither": ["l0.norm1", "l0.norm2"]}[keep])
    ids = M.tokens(cfg, 90)
    want = oracle(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(all_logits(eng, ids[:7]), want[:7], dtype)
    eng.close()


SIZES = [{"scale": 0.01}, {"scale": 1.5}, {"kv_heads": 1}, {"kv_heads": 6}, {"heads": 1, "kv_heads": 1}, {"heads": 9, "kv_heads": 1}, {"heads": 20, "kv_heads": 1},
         {"heads": 36, "kv_heads": 2}, {"dim": 1}, {"dim": 16}, {"dim": 33}, {"dim": 64}, {"dim": 130}, {"dim": 256}, {"dim": 270}, {"q_temp": None},
         {"q_temp": M.temp(2.0, 1)}, {"q_temp": M.temp(-0.2, 8)}, {"q_temp": M.temp(0.5, 7.5)}, {"q_temp": M.temp(0.5, 4000)}]
BIASED = [{"vdim": 1}, {"vdim": 70}, {"vdim": 150}, {"vdim": 300}, {"bias_max": 7, "rows": 12}, {"bias_max": 64, "rows": 16}, {"bias_max": 5000, "rows": 64},
          {"bias_max": 2, "rows": 2}, {"bias_max": 40, "rows": 9}, {"bias_max": 128, "rows": 200}]


@pytest.mark.parametrize("kind,change", [("shared", c) for c in SIZES] + [("biased", c) for c in SIZES + BIASED], ids=str)
def test_attention_sizes_and_constants(kind, change):
    cfg = M.config([(M.shared_kv if kind == "shared" else M.biased)(**{**dict(kv_heads=2, mlp=None), **change})], width=60)
    W = M.weights(cfg, seed=5, sharp=2.0)
    ids = M.tokens(cfg, 170)
    want = oracle(cfg, W, ids)
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, W, dtype)
        check(all_logits(eng, ids), want, dtype)
        check(in_portions(eng, ids, [9, 50], slot=1), want, dtype)
        eng.close()


@pytest.mark.parametrize("change", [dict(experts=1, top=1, groups=None), dict(experts=40, top=1, groups=(8, 1)), dict(experts=40, top=7, groups=(40, 9)),
                                    dict(experts=36, top=6, groups=(3, 2)), dict(experts=36, top=12, groups=(3, 1)), dict(groups=(1, 1)), dict(groups=(10, 10)),
                                    dict(experts=130, top=8, groups=(65, 40), ff=9), dict(scale=1.0), dict(scale=0.25), dict(ff=1), dict(ff=130),
                                    dict(shared=None), dict(shared=200)], ids=str)
def test_experts_sizes_and_constants(change):
    cfg = M.config([M.shared_kv(mlp=M.moe(**change))], width=72)
    W = M.silent(M.weights(cfg, seed=6), "l0.norm1")
    ids = M.tokens(cfg, 80)
    want = oracle(cfg, W, ids)
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, W, dtype)
        check(all_logits(eng, ids), want, dtype, 0.1)
        check(all_logits(eng, ids[:20]), want[:20], dtype, 0.1)
        check(in_portions(eng, ids[:12], [1, 3]), want[:12], dtype, 0.1)
        eng.close()


def test_router_without_a_scale_or_groups():
    cfg = M.config([M.shared_kv(mlp=M.moe(groups=None))])
    del cfg["layers"][0]["mlp"]["router"]["scale"]
    W = M.weights(cfg, seed=7)
    ids = M.tokens(cfg, 50)
    eng = engine(cfg, W, "float32")
    check(all_logits(eng, ids), oracle(cfg, W, ids), "float32")
    eng.close()


@BOTH
def test_groups_whose_scores_are_all_negative(dtype):
    """Kept groups with negative choice scores only: the others' experts must not come in between. The choice is wide apart."""
    cfg = M.config([M.biased(mlp=M.moe(experts=6, top=3, groups=(3, 2), shared=None))])
    W = M.weights(cfg, seed=8)
    W["l0.mlp.correction"] = M.bf16(np.array([-9.0, -3.0, -5.0, -7.0, -6.0, -8.0]))
    ids = M.tokens(cfg, 60)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), oracle(cfg, W, ids), dtype)
    check(all_logits(eng, ids[:5]), oracle(cfg, W, ids[:5]), dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("change", [dict(eps=0.3), dict(scale=0.11), dict(mult=1.0), dict(mult=0.2)], ids=str)
def test_constants_of_the_stream_and_layers_out(change, dtype):
    cfg = mixed_layers()
    cfg = M.config(cfg["layers"], vocab=90, width=76, **change)
    W = M.weights(cfg, seed=8)
    ids = M.tokens(cfg, 40)
    want, stream = L.forward(M.spelled(cfg), W, ids)
    eng = engine(cfg, W, dtype)
    eng.set_trace(True)
    check(all_logits(eng, ids), want, dtype)
    for i in range(len(cfg["layers"])):
        assert np.max(np.abs(eng.layer_out(i) - stream[i])) < TOL[dtype] * np.std(stream[i]) * 2, i
    eng.close()


def test_no_more_positions_than_the_table_has():
    cfg = M.config([M.shared_kv(mlp=None)], max_positions=40)
    W = M.weights(cfg, seed=9)
    ids = M.tokens(cfg, 41)
    eng = engine(cfg, W, "float32")
    check(all_logits(eng, ids[:40]), oracle(cfg, W, ids[:40]), "float32")
    with pytest.raises(Exception):
        eng.forward_mixed([(0, ids[40:], [0])])
    check(all_logits(eng, ids[:40]), oracle(cfg, W, ids[:40]), "float32")
    eng.close()


# ── whole prompts, decoding, portions, batches ──────────────────────────────
@BOTH
def test_varied_layers_prompt_and_decode(dtype):
    cfg = M.varied()
    W = M.weights(cfg, seed=1)
    ids = M.tokens(cfg, 150)
    want = oracle(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype, 0.25)
    check(in_portions(eng, ids[:100], [1]), want[:100], dtype, 0.25)
    eng.close()


@BOTH
@pytest.mark.parametrize("sizes", [[2], [3, 1], [15, 16, 17], [31, 2, 33], [40], [64, 5], [100, 1, 1]], ids=str)
def test_portions_of_any_size(sizes, dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=2, sharp=2.0)
    ids = M.tokens(cfg, 150)
    eng = engine(cfg, W, dtype)
    check(in_portions(eng, ids, sizes, slot=2), oracle(cfg, W, ids), dtype)
    eng.close()


@BOTH
def test_prompt_longer_than_a_chunk_of_the_engine(dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=2)
    ids = M.tokens(cfg, 150)
    want = oracle(cfg, W, ids)
    for rows in (1, 20, 37, 64):
        eng = engine(cfg, W, dtype, max_tokens=rows)
        check(all_logits(eng, ids), want, dtype)
        eng.close()


@BOTH
def test_mixed_batches_equal_each_request_alone(dtype):
    """Portions beside single tokens, requests left out of a step, slots and pages handed on; the pool holds no page more than the
    live requests need."""
    cfg = mixed_layers()
    W = M.weights(cfg, seed=4, sharp=2.0)
    lens = [120, 5, 77, 33, 60, 18, 1, 50]
    reqs = {r: M.tokens(cfg, n, seed=r) for r, n in enumerate(lens)}
    want = {r: oracle(cfg, W, t) for r, t in reqs.items()}
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
def test_freed_slots_and_pages_leave_nothing_behind(dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=9, sharp=3.0)
    eng = engine(cfg, W, dtype, max_batch=2, kv_pages=12)
    for seed, n in ((1, 180), (2, 3), (3, 1), (4, 50), (5, 16), (6, 17)):
        ids = M.tokens(cfg, n, seed)
        check(all_logits(eng, ids, slot=seed % 2), oracle(cfg, W, ids), dtype)
        eng.reset_cache(seed % 2)
    eng.close()


@BOTH
def test_first_tokens_and_long_decoding(dtype):
    cfg = mixed_layers()
    W = M.weights(cfg, seed=12, sharp=2.0)
    ids = M.tokens(cfg, 330)
    want = oracle(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    for n in (1, 2, 3):
        check(all_logits(eng, ids[:n]), want[:n], dtype)
    check(in_portions(eng, ids, [1]), want, dtype)
    eng.close()


@BOTH
def test_real_sized_layers(dtype):
    """Heads of the sizes that models have, keys split over blocks, biases and temperatures over a long context."""
    cfg = M.config([M.biased(heads=8, kv_heads=2, dim=128, vdim=128, bias_max=256, rows=32, q_temp=M.temp(0.3, 128), mlp=M.dense(300)),
                    M.shared_kv(heads=8, kv_heads=2, dim=128, q_temp=M.temp(0.3, 128), mlp=M.moe(experts=8, top=8, groups=(4, 4), ff=64, shared=96)),
                    M.biased(heads=2, kv_heads=2, dim=64, vdim=96, bias_max=1000, rows=64, mlp=None),
                    M.shared_kv(heads=12, kv_heads=1, dim=64, mlp=None)], width=264, max_positions=1500)
    W = M.weights(cfg, seed=13, sharp=2.0)
    ids = M.tokens(cfg, 1030)
    want = oracle(cfg, W, ids)
    eng = engine(cfg, W, dtype, max_ctx=1100, max_tokens=1100)
    check(all_logits(eng, ids), want, dtype)
    eng.reset_cache(0)
    eng.forward_mixed([(0, ids[:1000], [])])
    for a, b in ((1000, 1002), (1002, 1019), (1019, 1020), (1020, 1030)):
        check(eng.forward_mixed([(0, ids[a:b], places(b - a))]), want[a:b], dtype)
    eng.close()


@BOTH
def test_shared_pages_are_copied_before_they_are_written(dtype):
    """A prefix adopted from another sequence, cut in the middle of a page and continued differently."""
    cfg = mixed_layers()
    W = M.weights(cfg, seed=15)
    ids = M.tokens(cfg, 60)
    other = np.concatenate([ids[:40], M.tokens(cfg, 20, 5)])
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), oracle(cfg, W, ids), dtype)
    eng.adopt_prefix(1, [eng.slot_page(0, i) for i in range(3)])
    assert eng.truncate_cache(40, slot=1) == 40
    check(eng.forward_mixed([(1, other[40:], places(20))]), oracle(cfg, W, other)[40:], dtype)
    assert eng.truncate_cache(45, slot=0) == 45
    check(eng.forward_mixed([(0, ids[45:], places(15))]), oracle(cfg, W, ids)[45:], dtype)
    eng.close()


# ── one token, one distance, one step of the temperature ────────────────────
@BOTH
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_a_far_token_among_hundreds(kind, dtype):
    """The marker at every kind of place of a long context, found by prompts and by decoded tokens; without it the sink shows."""
    cfg, W = M.marker(kind, heads=12, kv_heads=4)
    eng = engine(cfg, W, dtype)
    n = 390
    for at in (0, 1, 15, 16, 63, 64, 200, 255, 256, 300, n - 2):
        ids = (1 + M.tokens(cfg, n, at) % 100).astype(np.uint32)
        ids[at] = M.MARK
        want = oracle(cfg, W, ids)
        gone = ids.copy()
        gone[at] = M.PLAIN
        assert M.error(oracle(cfg, W, gone)[-1:], want[-1:])[0] > 3 * TOL[dtype]
        check(all_logits(eng, ids), want, dtype)
        eng.reset_cache(1)
        eng.forward_mixed([(1, ids[:-1], [])])
        check(eng.forward_mixed([(1, ids[-1:], [0])]), want[-1:], dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("sink", [-20.0, 6.0, 15.0])
def test_sinks_of_any_size(kind, sink, dtype):
    """From one that counts nothing to one that takes all: the mixture then vanishes before the norm sees it."""
    cfg, W = M.marker(kind, sink=sink)
    cfg["norm"]["eps"] = 1e-3
    ids = (1 + M.tokens(cfg, 200, 3) % 100).astype(np.uint32)
    ids[70] = M.MARK
    want = oracle(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(in_portions(eng, ids, [1, 20, 50, 60], slot=1), want, dtype)
    eng.close()


@BOTH
@pytest.mark.parametrize("at", [0, 3, 9, 10, 40, 150, 260])
def test_one_distance_stands_out(at, dtype):
    """Buckets just inside and just outside their edges, in prompts and in decoding, at page borders and between them."""
    cfg, W = M.one_distance(at)
    ids = M.tokens(cfg, 300)
    want = oracle(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(in_portions(eng, ids, [200, 1, 1, 1, 14, 1, 1, 33], slot=1), want, dtype)
    first = next(n for n in range(at + 1) if L.bucket(n, 20, 200) == L.bucket(at, 20, 200))
    for p in {max(first - 1, 0), first, first + 1}:
        eng.reset_cache(2)
        if p:
            eng.forward_mixed([(2, ids[:p], [])])
        check(eng.forward_mixed([(2, ids[p:p + 1], [0])]), want[p:p + 1], dtype)
    eng.close()


@BOTH
def test_steps_of_the_temperature(dtype):
    """A factor that grows so much that a token on the wrong side of a step shows."""
    cfg = M.config([M.shared_kv(q_temp=M.temp(3.0, 16), mlp=None), M.biased(q_temp=M.temp(2.0, 33), mlp=None)], width=72)
    W = M.weights(cfg, seed=16)
    ids = M.tokens(cfg, 140)
    want = oracle(cfg, W, ids)
    eng = engine(cfg, W, dtype)
    check(all_logits(eng, ids), want, dtype)
    check(in_portions(eng, ids, [1]), want, dtype)
    eng.close()


# ── generation through the framework's entry points ─────────────────────────
def oracle_greedy(cfg, W, prompt, n):
    ids, gaps = list(prompt), []
    for _ in range(n):
        z = oracle(cfg, W, ids)[-1]
        top = np.sort(z)[-2:]
        gaps.append(top[1] - top[0])
        ids.append(int(np.flatnonzero(z == z.max())[-1]))
    gaps = np.asarray(gaps)
    return ids[len(prompt):], int(np.argmax(gaps < 1e-3)) if (gaps < 1e-3).any() else n  # up to a near tie


def test_greedy_generation_through_the_scheduler():
    cfg = M.config([M.biased(), M.shared_kv(), M.biased(mlp=M.moe())], vocab=133, width=76)
    W = M.weights(cfg, seed=30, loud=2.0)
    prompts = [M.tokens(cfg, n, seed=50 + n) for n in (3, 40, 17, 90, 64)]
    prompts.append(np.concatenate([prompts[4], M.tokens(cfg, 5, 99)]))   # starts like the one before: its pages are shared
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
    assert b.stats().shared_tokens >= 64
    b.close()
    first = eng.forward_mixed([(0, prompts[0], [len(prompts[0]) - 1])], want_argmax=True)
    toks = [int(first[0])] + eng.decode_greedy(first, [0], 11)[:, 0].tolist()
    want, upto = oracle_greedy(cfg, W, prompts[0], 12)
    assert toks[:upto] == want[:upto]
    eng.close()


def test_bf16_generation_does_not_depend_on_the_batch_or_on_graphs():
    cfg = mixed_layers()
    W = M.weights(cfg, seed=31, loud=2.0)
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
        z = oracle(cfg, W, ids[:-1])[len(p):]
        for seq in (alone, together[:, i]):              # every pick is a maximum within the tolerance, up to where the two part
            same = int(np.argmax(seq != alone)) if (seq != alone).any() else 40
            picked = z[np.arange(same), seq[:same].astype(int)]
            assert np.all(z[:same].max(-1) - picked < 6 * TOL["bfloat16"] * z.std())
            assert same >= 10 or z[same].max() - z[same][int(seq[same])] < 6 * TOL["bfloat16"] * z.std()
    eng.close()


def test_speculative_loops():
    from sapient_b200 import speculative

    cfg = mixed_layers()
    W = M.weights(cfg, seed=32, loud=2.0)
    other = M.config([M.biased()], vocab=cfg["vocab"], width=40)
    p = M.tokens(cfg, 20)
    want, upto = oracle_greedy(cfg, W, p, 20)
    a = engine(cfg, W, "float32", max_batch=1)
    b = engine(other, M.weights(other, seed=33), "float32", max_batch=1)
    toks, _ = speculative.generate_greedy_device(a, b, p, 20, k=3)
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
    want = oracle(cfg, W, ids)
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
    W = M.weights(cfg, seed=41, loud=2.0)
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
