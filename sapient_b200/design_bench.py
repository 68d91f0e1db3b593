"""Throughput of layer-plan designs beside the framework's closest GGUF block at equal size (`bench.py --design NAME`).

Per size: the design with random bf16 weights, and a Llama block of the same width, heads, layers and ACTIVE feed-forward
weights in Q8_0 — prefill of one prompt, greedy decode at batch 1 and 32, device time by
CUDA events, and for each family of kernels of a decode step and of a prefill its device time, algorithmic bytes and flops
and the fraction of the roofline max(bytes / copy bandwidth, flops / GEMM rate) that is. Weights exceed L2 at every size.
"""
from __future__ import annotations

import json

import numpy as np

from . import synth
from .configs_bench import _engine, _timed
from .engine import ForwardEngine

# design -> size -> keywords of its configuration
LEPALORN = {
    "2b": dict(layers=6, width=2048, heads=16, dim=128, rot=64, vdim=128, rank=512, window=1024, experts=64, top=6, ff=1408, shared_ff=2816,
               vocab=32768, shared_latent_from=3),
    "8b": dict(layers=4, width=4096, heads=32, dim=128, rot=64, vdim=128, rank=512, window=4096, experts=32, top=4, ff=2048, shared_ff=2048,
               vocab=32768, shared_latent_from=2),
}
_PATTERN = ["general_delta", "general_delta", "attention", "lightning"]
TEDELIX = {
    "2b": dict(layers=_PATTERN * 2, width=2048, heads=16, kv_heads=4, dim=128, vdim=128, state_heads=32, state_dim=64, state_vdim=64, window=1024, ff=6144, vocab=32768),
    "8b": dict(layers=_PATTERN, width=4096, heads=32, kv_heads=8, dim=128, vdim=128, state_heads=64, state_dim=64, state_vdim=64, window=2048, ff=12288, vocab=32768),
}
TEDELIX_RANK = 64  # of the decay logits
# dense and active expert feed-forwards of a size have equal weights
FATILIX = {
    "2b": dict(layers=["attention_2", "attention"] * 3, width=2048, heads=16, kv_heads=4, dim=128, vdim=128, ff=9216, experts=64, top=8, groups=8, keep=4,
               expert_ff=512, shared_ff=2048, vocab=32768, max_positions=4096, bias_max=512),
    "8b": dict(layers=["attention_2", "attention"] * 2, width=4096, heads=32, kv_heads=8, dim=128, vdim=128, ff=18432, experts=32, top=4, groups=4, keep=2,
               expert_ff=2048, shared_ff=4096, vocab=32768, max_positions=4096, bias_max=512),
}
_ATTENTION = dict(conv=4, keep_first=4, vocab=32768)
REVELIX = {
    "2b": dict(layers=["retention", "parallel", "parallel"] * 2, width=2048, heads=16, kv_heads=4, dim=128, vdim=128, state_heads=16, state_dim=64, state_vdim=64,
               retention_heads=16, retention_dim=128, retention_vdim=128, window=1024, ff=6144, **_ATTENTION),
    "8b": dict(layers=["retention", "parallel", "parallel", "retention"], width=4096, heads=32, kv_heads=8, dim=128, vdim=128, state_heads=32, state_dim=64, state_vdim=64,
               retention_heads=32, retention_dim=128, retention_vdim=128, window=2048, ff=12288, **_ATTENTION),
}


def lepalorn_llama(s: dict) -> dict:
    """Same width, heads, layers and active feed-forward width."""
    return _llama(s, s["layers"], s["heads"], s["top"] * s["ff"] + s["shared_ff"])


def tedelix_llama(s: dict) -> dict:
    """Same width, heads, layers and feed-forward weights (three matrices for two)."""
    return _llama(s, len(s["layers"]), s["kv_heads"], 2 * s["ff"] // 3)


def fatilix_llama(s: dict) -> dict:
    """Same width, heads, layers and active feed-forward weights."""
    return _llama(s, len(s["layers"]), s["kv_heads"], s["top"] * s["expert_ff"] + s["shared_ff"])


def revelix_llama(s: dict) -> dict:
    """Same width, heads, layers and, over all layers, feed-forward weights."""
    ff = 2 * s["ff"] * s["layers"].count("parallel") / (3 * len(s["layers"]))
    return _llama(s, len(s["layers"]), s["kv_heads"], round(ff / 256) * 256)


def _llama(s: dict, layers: int, kv_heads: int, ffn: int) -> dict:
    return dict(arch="llama", n_layers=layers, hidden=s["width"], n_heads=s["heads"], n_kv_heads=kv_heads, head_dim=128, ffn=ffn, vocab=s["vocab"],
                norm_eps=1e-5, rope_theta=1e4, tied=False)


def lepalorn_model(s: dict):
    cfg = synth.lepalorn_config(**s)
    return cfg, synth.lepalorn_weights(cfg, seed=11, device="cuda")


def tedelix_model(s: dict):
    cfg = synth.tedelix_config(**s)
    return cfg, synth.tedelix_weights(cfg, seed=11, rank=TEDELIX_RANK, device="cuda")


def fatilix_model(s: dict):
    cfg = synth.fatilix_config(**s)
    return cfg, synth.fatilix_weights(cfg, seed=11, device="cuda")


def revelix_model(s: dict):
    cfg = synth.revelix_config(**s)
    return cfg, synth.revelix_weights(cfg, seed=11, device="cuda")


def design_engine(cfg: dict, W: dict, **kw):
    import torch

    W = {k: v.cpu() for k, v in W.items()}
    torch.cuda.empty_cache()
    eng = ForwardEngine.from_config(cfg, W, **kw)
    stream = torch.cuda.Stream()
    torch.cuda.set_stream(stream)
    eng.set_stream(stream.cuda_stream)
    return eng, stream


def llama_engine(shape: dict, max_ctx: int, **kw):
    import torch

    cfg, W = synth.build_model(shape, seed=12, device="cuda", max_ctx=max_ctx, dtype=synth.Q8_0)
    W = synth.weights_to_numpy(W)
    torch.cuda.empty_cache()
    eng, stream = _engine(cfg, W, **kw)
    return eng, stream


def _distinct(experts: int, top: int, rows: int) -> float:
    """Expected number of experts that at least one of `rows` tokens chooses (uniform choice)."""
    return experts * (1.0 - (1.0 - top / experts) ** rows)


def _pairs(n: int, window: int) -> int:
    """(query, key) pairs of a causal prompt of n tokens under a sliding window."""
    w = min(n, window)
    return w * (w + 1) // 2 + (n - w) * w


def lepalorn_work(s: dict, rows: int, ctx: int, prefill: bool) -> dict:
    """Algorithmic (bytes, flops) of one step by kernel family. Prefill: one sequence of `rows` tokens; decode: `rows`
    sequences with `ctx` cached tokens each."""
    L, W, H, D, R, V, K, E = s["layers"], s["width"], s["heads"], s["dim"], s["rot"], s["vdim"], s["rank"], s["experts"]
    own = s["shared_latent_from"] + 1 if s["shared_latent_from"] is not None else L
    dense = L * (H * (D + R) * W + H * W + H * (D + V) * K + W * H * V + (E + 1) * W + 3 * s["shared_ff"] * W) + own * (K + R) * W
    active = L * 3 * s["ff"] * W
    used = _distinct(E, s["top"], rows)
    head = s["vocab"] * W
    keys = _pairs(rows, s["window"]) if prefill else rows * min(ctx, s["window"])
    per_pair = 2 * H * (D + R + V) if prefill else 2 * H * (K + R + K)
    return {"gemv": (2 * (dense + active * used + head), 2 * rows * (dense + active * s["top"]) + 2 * head * (1 if prefill else rows)),
            "attention": (L * 2 * (K + R) * (rows if prefill else keys), L * per_pair * keys),
            # residual + norm after the mixer; mixture, norm, residual and depth average (all results so far) after the experts
            "norm": (rows * W * sum(14 + 4 * s["top"] + 18 + 4 * (i + 1) for i in range(L)), 0),
            "rope_kv": (rows * 6 * (L * H * (D + R) + own * (K + R)), 0)}


def tedelix_work(s: dict, rows: int, ctx: int, prefill: bool) -> dict:
    """The same. State mixers: what enters them (f32 rows) and leaves, and the states read and written once per step; bytes only,
    their arithmetic is not tensor-core work."""
    W, H, G, D, V, HS, DS, VS, F = (s[k] for k in ("width", "heads", "kv_heads", "dim", "vdim", "state_heads", "state_dim", "state_vdim", "ff"))
    n = {t: s["layers"].count(t) for t in ("attention", "lightning", "general_delta")}
    L, hd, hv, R = len(s["layers"]), HS * DS, HS * VS, TEDELIX_RANK
    mats = 2 * L * F * W + n["attention"] * (H * D + G * (D + V) + H * V) * W + n["lightning"] * (2 * hd + 3 * hv) * W
    mats += n["general_delta"] * ((6 * hd + R) * W + hd * R)
    head = s["vocab"] * W
    keys = _pairs(rows, s["window"]) if prefill else rows * min(ctx, s["window"])
    seqs = 1 if prefill else rows
    states = 8 * seqs * (n["lightning"] * HS * DS * VS + n["general_delta"] * HS * DS * DS)
    return {"gemv": (2 * (mats + head), 2 * rows * mats + 2 * head * (1 if prefill else rows)),
            "attention": (n["attention"] * 2 * (G * (D + V) * (rows if prefill else keys) + rows * H * (D + V)), n["attention"] * 2 * H * (D + V) * keys),
            "state": (states + rows * (n["lightning"] * (4 * (2 * hd + 2 * hv) + 2 * hv) + n["general_delta"] * (4 * 5 * hd + 2 * hd)), 0),
            "norm": (rows * W * 6 * L, 0), "rope_kv": (rows * n["attention"] * 6 * (H * D + G * (D + V)), 0)}


def fatilix_work(s: dict, rows: int, ctx: int, prefill: bool) -> dict:
    """The same. Cached rows are read once: keys and values, or keys that are the values with their f32 factor; queries, mixtures
    and gate logits move once per token."""
    W, H, G, D, V, E, top = (s[k] for k in ("width", "heads", "kv_heads", "dim", "vdim", "experts", "top"))
    n = {t: s["layers"].count(t) for t in ("attention", "attention_2")}
    L = len(s["layers"])
    mats = L * (H * (D + 2 * V) + G * D) * W + n["attention_2"] * (G * V + 2 * s["ff"]) * W + n["attention"] * (E + 3 * s["shared_ff"]) * W
    active, used, head = n["attention"] * 3 * s["expert_ff"] * W, _distinct(E, top, rows), s["vocab"] * W
    keys = _pairs(rows, 1 << 30) if prefill else rows * ctx
    cached = G * (n["attention"] * (2 * D + 4) + n["attention_2"] * 2 * (D + V))
    return {"gemv": (2 * (mats + active * used + head), 2 * rows * (mats + active * top) + 2 * head * (1 if prefill else rows)),
            "attention": (cached * (rows if prefill else keys) + L * rows * H * (2 * D + 6 * V), L * 2 * H * (D + V) * keys),
            "norm": (rows * W * (14 * L + n["attention_2"] * 14 + n["attention"] * (14 + 4 * top)), 0),
            "rope_kv": (rows * (L * 6 * H * D + G * (n["attention"] * (6 * D + 4) + n["attention_2"] * 6 * (D + V))), 0)}


def revelix_work(s: dict, rows: int, ctx: int, prefill: bool) -> dict:
    """The same. Attention: scores, mixed weights and mixtures; states as for Tedelix; the stream's norms are part of the products."""
    W, H, G, D, V, F = (s[k] for k in ("width", "heads", "kv_heads", "dim", "vdim", "ff"))
    P, R = s["layers"].count("parallel"), s["layers"].count("retention")
    hd, hv, rd, rv = (s[a] * s[b] for a, b in (("state_heads", "state_dim"), ("state_heads", "state_vdim"), ("retention_heads", "retention_dim"),
                                               ("retention_heads", "retention_vdim")))
    qkv = H * D + G * (D + V)
    mats = P * (qkv + H * V + 2 * hd + 2 * hv + 2 * F) * W + R * (2 * rd + 3 * rv) * W
    head = s["vocab"] * W
    span = s["window"] + s["keep_first"]
    keys = _pairs(rows, span) if prefill else rows * min(ctx, span)
    seqs = 1 if prefill else rows
    states = 8 * seqs * (P * hd * s["state_vdim"] + R * rd * s["retention_vdim"])
    return {"gemv": (2 * (mats + head), 2 * rows * mats + 2 * head * (1 if prefill else rows)),
            "attention": (P * 2 * (G * (D + V) * (rows if prefill else keys) + rows * H * (D + V)), P * 2 * H * (D + V + H) * keys),
            "state": (states + rows * (P * (4 * (2 * hd + hv) + 2 * hv) + R * (4 * (2 * rd + 2 * rv) + 2 * rv)), 0),
            "norm": ((1 if prefill else rows) * W * 6, 0), "rope_kv": (rows * P * 6 * qkv, 0)}


def llama_work(c: dict, rows: int, ctx: int, prefill: bool) -> dict:
    q, kv = c["n_heads"] * c["head_dim"], c["n_kv_heads"] * c["head_dim"]
    mats = c["n_layers"] * (2 * (q + kv) * c["hidden"] + 3 * c["ffn"] * c["hidden"])
    head = c["vocab"] * c["hidden"]
    keys = _pairs(rows, 1 << 30) if prefill else rows * ctx
    return {"gemv": (34 / 32 * (mats + head), 2 * rows * mats + 2 * head * (1 if prefill else rows)),
            "attention": (c["n_layers"] * 2 * 2 * kv * (rows if prefill else keys), c["n_layers"] * 4 * q * keys),
            "norm": (rows * c["hidden"] * c["n_layers"] * 2 * 8, 0), "rope_kv": (rows * c["n_layers"] * (8 * q + 6 * 2 * kv), 0)}


# design -> (sizes, model of a size, its work, the Llama block of equal size)
DESIGNS = {"lepalorn": ("Lepalorn", LEPALORN, lepalorn_model, lepalorn_work, lepalorn_llama),
           "tedelix": ("Tedelix", TEDELIX, tedelix_model, tedelix_work, tedelix_llama),
           "fatilix": ("Fatilix", FATILIX, fatilix_model, fatilix_work, fatilix_llama),
           "revelix": ("Revelix", REVELIX, revelix_model, revelix_work, revelix_llama)}


def _families(ms: dict, work: dict, peaks: dict) -> dict:
    out = {}
    for f, t in ms.items():
        if t <= 0:
            continue
        out[f] = {"ms": round(t, 4)}
        if f in work:
            b, fl = work[f]
            floor = max(b / (peaks["hbm_gbs"] * 1e9), fl / (peaks["bf16_tflops"] * 1e12)) * 1e3
            out[f].update(roofline_ms=round(floor, 4), frac=round(floor / t, 3))
    return out


def measure(eng, stream, vocab: int, work, prompt: int, ctx: int, batch: int, steps: int, peaks: dict, fast: bool = False) -> dict:
    rng = np.random.default_rng(0)
    ids = rng.integers(0, vocab, prompt).astype(np.uint32)
    if fast:
        eng.set_large_m_gemm(1)
    res = {}
    for _ in range(3):
        eng.reset_cache(0)
        eng.forward_slot(0, ids)
    times = []
    for _ in range(5):
        eng.reset_cache(0)
        times.append(_timed(stream, lambda: eng.forward_slot(0, ids)))
    ms = sorted(times)[len(times) // 2]
    eng.reset_cache(0)
    eng.profile_read()
    eng.set_profile(True)
    eng.forward_slot(0, ids)
    fam = {k: v[0] for k, v in eng.profile_read().items()}
    eng.set_profile(False)
    res["prefill"] = {"tokens": prompt, "ms": round(ms, 3), "tokens_per_s": round(prompt / ms * 1e3), "families": _families(fam, work(prompt, 0, True), peaks)}
    for b in (1, batch):
        eng.reset_cache()
        for i in range(b):
            eng.forward_slot(i, rng.integers(0, vocab, ctx).astype(np.uint32))
        slots = list(range(b))
        first = rng.integers(0, vocab, b).astype(np.uint32)
        toks = eng.decode_greedy(first, slots, 8)
        ms = _timed(stream, lambda: eng.decode_greedy(toks[-1], slots, steps, fetch=False)) / steps
        eng.synchronize()
        todo = work(b, ctx, False)
        fam = {f: eng.time_families(f, b, 20) for f in eng.PROFILE_FAMILIES if f != "state" or f in todo}
        res[f"decode_b{b}"] = {"ctx": ctx, "ms_per_step": round(ms, 4), "tokens_per_s": round(b / ms * 1e3), "families": _families(fam, todo, peaks)}
    return res


def run(design: str, peaks: dict, sizes=None, prompt: int = 2048, ctx: int = 1024, batch: int = 32, steps: int = 32, designs_only: bool = False) -> dict:
    if design.lower() not in DESIGNS:
        raise SystemExit(f"no such design: {design}")
    title, all_sizes, model, design_work, llama_like = DESIGNS[design.lower()]
    out = {"design": title, "data": "synthetic random weights", "peaks": {k: peaks[k] for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    kw = dict(max_batch=batch, max_tokens=prompt, kv_pages=(max(prompt, 0) + batch * (ctx + 256)) // 16)
    for name in sizes or all_sizes:
        s = all_sizes[name]
        r = {"config": s}
        eng, stream = design_engine(*model(s), max_ctx=prompt + ctx, **kw)
        r["design"] = measure(eng, stream, s["vocab"], lambda a, c, p: design_work(s, a, c, p), prompt, ctx, batch, steps, peaks)
        eng.close()
        if not designs_only:
            shape = llama_like(s)
            for tag, fast in (("llama_q8_0", False), ("llama_q8_0_fp16_operands", True)):
                eng, stream = llama_engine(shape, prompt + ctx, **kw)
                r[tag] = measure(eng, stream, s["vocab"], lambda a, c, p: llama_work(shape, a, c, p), prompt, ctx, batch, steps, peaks, fast)
                eng.close()
        out["sizes"][name] = r
        print(json.dumps({name: r}), flush=True)
    return out
