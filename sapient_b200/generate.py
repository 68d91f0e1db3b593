"""Generation from token ids on the command line (tokenizers are the caller's):

    python -m sapient_b200.generate --model model.gguf --prompt 1,15043,29892 --max-new 32
    python -m sapient_b200.generate --model model_dir --dtype bfloat16 --prompt 5,6,7 --prompt 9 --temperature 0.8

--model: a GGUF file, or a directory with config.json and model.safetensors. Prompts run together; one JSON line each,
in order. Greedy requests go through the continuous-batching scheduler, sampled ones through mixed steps with the host
sampler (softmax of logits / temperature, inverse-CDF draw: crates/sapient-generate/src/speculative.rs:635-690).
"""
from __future__ import annotations

import argparse
import json
import os

import numpy as np

from .batching import ContinuousBatcher
from .engine import ForwardEngine
from .speculative import sample_from_probs, softmax


def load(path: str, dtype: str = "bfloat16", max_ctx: int = 4096, max_batch: int = 1, device: int = 0) -> ForwardEngine:
    """An engine for a GGUF file or a model directory; the registry chooses the model."""
    if os.path.isdir(path):
        return ForwardEngine.from_pretrained(path, dtype=dtype, max_ctx=max_ctx, max_batch=max_batch, device=device)
    return ForwardEngine.from_gguf(path, device=device, max_ctx=max_ctx, max_batch=max_batch)


def generate_greedy(eng: ForwardEngine, prompts, max_new: int, eos=()) -> list:
    b = ContinuousBatcher(eng)
    try:
        ids = [b.submit(p, max_new, eos) for p in prompts]
        b.run()
        return [[int(t) for t in b.poll(i)[0]] for i in ids]
    finally:
        b.close()


def generate_sampled(eng: ForwardEngine, prompts, max_new: int, temperature: float, seed: int = 0, eos=()) -> list:
    """All prompts as one mixed step, then one token of every unfinished sequence per step."""
    rng = np.random.default_rng(seed)
    out = [[] for _ in prompts]
    feed = {i: list(p) for i, p in enumerate(prompts)}
    while feed:
        order = list(feed)
        logits = eng.forward_mixed([(i, feed[i], [len(feed[i]) - 1]) for i in order])
        feed = {}
        for i, z in zip(order, logits):
            t = sample_from_probs(softmax(z / np.float32(temperature)), float(rng.random(dtype=np.float32)))
            out[i].append(t)
            if t in eos or len(out[i]) >= max_new:
                eng.reset_cache(i)
            else:
                feed[i] = [t]
    return out


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(ForwardEngine.COMPUTE), help="compute type of a model directory")
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be repeated")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--eos", default="", help="comma-separated ids that end a sequence")
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--max-ctx", type=int, default=4096)
    a = ap.parse_args()
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    eos = [int(t) for t in a.eos.split(",") if t]
    eng = load(a.model, a.dtype, a.max_ctx, len(prompts))
    toks = generate_sampled(eng, prompts, a.max_new, a.temperature, a.seed, eos) if a.temperature > 0 else generate_greedy(eng, prompts, a.max_new, eos)
    for p, t in zip(prompts, toks):
        print(json.dumps({"prompt": p, "tokens": t}), flush=True)
    eng.close()


if __name__ == "__main__":
    main()
