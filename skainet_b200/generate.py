"""Generation over a loaded decoder: prompts of any lengths enter slots as they become free, are prefilled one by one
and then decode together; greedy or temperature sampling.

    python -m skainet_b200.generate --model DIR --prompt 5,17,3 [--prompt ...] [--max-new 16] [--temperature T]
"""
from __future__ import annotations

import argparse
from typing import List, Optional, Sequence

import numpy as np


def sample(logits: np.ndarray, temperature: float, rng) -> int:
    """One id from a row of logits (temperature 0: the first maximum)."""
    if temperature <= 0:
        return int(np.argmax(logits))
    z = logits.astype(np.float64) / temperature
    p = np.exp(z - z.max())
    return int(rng.choice(p.size, p=p / p.sum()))


def generate(model, prompts: Sequence[Sequence[int]], max_new: int, temperature: float = 0.0, seed: int = 0,
             stop: Optional[int] = None) -> List[List[int]]:
    """New ids for every prompt.  Slots 0 .. max_seqs - 1 of `model` are used; a finished sequence frees its slot for
    the next waiting prompt, and neighbouring slots that decode share a step."""
    rng = np.random.default_rng(seed)
    out: List[List[int]] = [[] for _ in prompts]
    waiting = list(range(len(prompts)))
    slots: List[Optional[int]] = [None] * model.max_seqs     # request in each slot
    fed = [0] * model.max_seqs                               # id that the slot takes next

    def take(slot, next_id):
        req = slots[slot]
        out[req].append(next_id)
        fed[slot] = next_id
        if len(out[req]) >= max_new or next_id == stop:
            slots[slot] = None
            model.reset(slot)

    if max_new < 1:
        return out
    while waiting or any(s is not None for s in slots):
        for i in range(model.max_seqs):
            while slots[i] is None and waiting:
                slots[i] = waiting.pop(0)
                model.reset(i)
                p = prompts[slots[i]]
                nxt, lg = model.forward(p, seq=i, want=[len(p) - 1] if temperature > 0 else (), want_next=temperature <= 0)
                take(i, int(nxt[0]) if temperature <= 0 else sample(lg[0], temperature, rng))
        i = 0
        while i < model.max_seqs:
            if slots[i] is None:
                i += 1
                continue
            n = 1
            while i + n < model.max_seqs and slots[i + n] is not None and n < 64:
                n += 1
            tok = np.asarray(fed[i:i + n], dtype=np.int32).reshape(n, 1)
            nxt, lg = model.forward(tok, seq=i, want=range(n) if temperature > 0 else (), want_next=temperature <= 0)
            for k in range(n):
                take(i + k, int(nxt[k]) if temperature <= 0 else sample(lg[k], temperature, rng))
            i += n
    return out


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m skainet_b200.generate", description="Generate token ids with a model folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be given several times")
    ap.add_argument("--max-new", type=int, default=16)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--stop", type=int, default=None, help="id that ends a sequence")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-seqs", type=int, default=8)
    ap.add_argument("--max-tokens", type=int, default=1024, help="most tokens of one step")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    from . import _ffi, build, registry
    from .tensor import Context
    _ffi.use(build.build_family(registry.architecture_of(registry.read_config(a.model)).family))
    prompts = [[int(x) for x in p.split(",")] for p in a.prompt]
    ctx = Context(a.device)
    model = registry.load_model(ctx, a.model, max_seqs=min(a.max_seqs, len(prompts)), max_tokens=a.max_tokens,
                                max_ctx=max(len(p) for p in prompts) + a.max_new, dtype=a.dtype)
    for ids in generate(model, prompts, a.max_new, a.temperature, a.seed, a.stop):
        print(",".join(map(str, ids)))
    model.close()
    ctx.close()


if __name__ == "__main__":
    main()
