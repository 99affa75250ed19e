"""Generation: a batch of prompts through an engine of the registry.

`generate` admits prompts as slots become free, feeds each in portions, decodes all live sequences together, one token
per step, and retires them as they finish.

    python -m reimagined_b200.generate --model DIR --prompt 5,17,3 --prompt 8,9 --tokens 32
"""
from __future__ import annotations

import argparse
import json
from collections import deque
from typing import List, Optional, Sequence

import torch

from . import registry


def sample(logits: torch.Tensor, temperature: float = 0.0, top_k: int = 0, top_p: float = 1.0,
           generator: Optional[torch.Generator] = None) -> torch.Tensor:
    """Token ids [n] from logits [n, vocab]; temperature 0 is greedy (the lowest id wins a tie)."""
    if temperature <= 0.0:
        return logits.argmax(dim=-1)
    z = logits / temperature
    if top_k > 0:
        kth = z.topk(min(top_k, z.shape[-1]), dim=-1).values[..., -1:]
        z = z.masked_fill(z < kth, float("-inf"))
    p = z.softmax(dim=-1)
    if top_p < 1.0:
        ordered, index = p.sort(dim=-1, descending=True)
        drop = ordered.cumsum(dim=-1) - ordered >= top_p          # the most probable token always stays
        p = torch.zeros_like(p).scatter(-1, index, ordered.masked_fill(drop, 0.0))
    return torch.multinomial(p, 1, generator=generator).squeeze(-1)


def generate(engine, prompts: Sequence[Sequence[int]], max_new: int, stop: Sequence[int] = (), temperature: float = 0.0,
             top_k: int = 0, top_p: float = 1.0, seed: Optional[int] = None) -> List[List[int]]:
    """The new tokens of every prompt (a stop token ends a sequence and is included)."""
    for p in prompts:
        if not len(p):
            raise ValueError("a prompt needs at least one token")
        if len(p) + max_new - 1 > engine.capacity:
            raise ValueError(f"prompt of {len(p)} + {max_new} new tokens does not fit the capacity {engine.capacity}")
    out: List[List[int]] = [[] for _ in prompts]
    if max_new <= 0:
        return out
    gen = None
    if temperature > 0.0:
        gen = torch.Generator(device="cuda")
        gen.manual_seed(0 if seed is None else seed)
    stops, waiting, live = set(stop), deque(range(len(prompts))), {}

    def accept(requests, logits):
        for r, t in zip(requests, sample(logits, temperature, top_k, top_p, gen).tolist()):
            out[r].append(t)
            if len(out[r]) >= max_new or t in stops:
                engine.close(live.pop(r))

    while waiting or live:
        while waiting and len(live) < engine.slots:
            r = waiting.popleft()
            live[r] = engine.open()
            accept([r], engine.feed(live[r], prompts[r]))
        if live:
            requests = list(live)
            accept(requests, engine.step([live[r] for r in requests], [[out[r][-1]] for r in requests]))
    return out


def main() -> None:
    ap = argparse.ArgumentParser(description="generate token ids from prompts of token ids")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--prompt", action="append", required=True, help="token ids with commas between them; may be repeated")
    ap.add_argument("--tokens", type=int, default=32, help="most new tokens per prompt")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--batch", type=int, default=0, help="sequences decoded together (default: all prompts)")
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--stop", default="", help="token ids that end a sequence")
    args = ap.parse_args()
    ids = lambda text: [int(t) for t in text.split(",") if t.strip()]
    prompts = [ids(p) for p in args.prompt]
    engine = registry.load(args.model, args.dtype, slots=args.batch or len(prompts),
                           capacity=max(len(p) for p in prompts) + args.tokens)
    for p, new in zip(prompts, generate(engine, prompts, args.tokens, ids(args.stop), args.temperature, args.top_k,
                                        args.top_p, args.seed)):
        print(json.dumps({"prompt": p, "tokens": new}))


if __name__ == "__main__":
    main()
