"""Model registry: config.json's "architecture" -> the engine that serves it.

Every engine offers the same few calls to generation and replay: `open() -> slot`, `feed(slot, tokens, want) ->
logits`, `step(slots, tokens) -> logits` (one or more tokens of several sequences), `close(slot)`, and the attributes
`vocab`, `slots`, `capacity`.  An entry also names the shared library it needs, so that only that one is built.
"""
from __future__ import annotations

import os
from typing import Callable, Dict, NamedTuple, Tuple

from . import build
from .checkpoint import read_config


class Entry(NamedTuple):
    library: str                  # key of build.LIBRARIES
    dtypes: Tuple[str, ...]
    load: Callable                # (folder, config, dtype, slots, capacity) -> engine


def _load_stack(folder, cfg, dtype, slots, capacity):
    from . import stack
    return stack.load(folder, dtype, slots, capacity, cfg)


def _load_hybrid(folder, cfg, dtype, slots, capacity):
    import numpy as np
    from .decode import DecodeSession
    with np.load(os.path.join(folder, "params.npz")) as f:
        return DecodeSession(dict(f), capacity)


MODELS: Dict[str, Entry] = {
    "Guselix": Entry("stack", ("bfloat16", "float32"), _load_stack),
    "Goguvik": Entry("stack", ("bfloat16", "float32"), _load_stack),
    # the Mamba-2 / attention hybrid on ternary weights: params.npz holds DecodeEngine's parameter set
    "JambaHybrid": Entry("ternary", ("bfloat16",), _load_hybrid),
}


def entry(folder: str) -> Tuple[Entry, dict]:
    cfg = read_config(folder)
    name = cfg.get("architecture")
    if name not in MODELS:
        raise ValueError(f"no model named {name!r}; known: {', '.join(sorted(MODELS))}")
    return MODELS[name], cfg


def load(folder: str, dtype: str = "bfloat16", slots: int = 1, capacity: int = 1024):
    """Builds the library the model needs if it is not up to date, and opens the engine."""
    e, cfg = entry(folder)
    if dtype not in e.dtypes:
        raise ValueError(f"{cfg['architecture']} does not run in {dtype}")
    build.build(libraries=(e.library,))
    return e.load(folder, cfg, dtype, slots, capacity)
