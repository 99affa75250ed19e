"""Configurations, weights and error measures shared by the layer-stack tests."""
import numpy as np


def delta(heads, dim, mlp=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=500.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot_dim}}}


def attention(heads, kv_heads, dim, vdim, scale, diff, coef, every, mlp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "q_temp": {"coef": coef, "every": every}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def ff(n):
    return {"kind": "dense", "ff": n}


def config(layers, width, vocab, scale=0.7, eps=1e-5):
    return {"architecture": "Guselix", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


def stream_config(layers, width, vocab, streams, eps=1e-5):
    return {"architecture": "Goguvik", "layers": layers, "norm": {"eps": eps}, "streams": streams, "vocab": vocab, "width": width}


# sizes that fit no tile, vector or warp; feed-forwards after either mixer
ODD = config([latent(5, 20, 12, 28, 36, 44, 0.31, 90.0, ff(50)), delta(3, 22, ff(37)), latent(2, 6, 2, 10, 7, 9, 0.6, 7.0)],
             width=90, vocab=131)
# sizes the tensor-core kernels take; the value size differs from the key size either way
EVEN = config([delta(3, 64), latent(3, 48, 16, 80, 64, 80, 0.2, 1e4, ff(200)), delta(2, 40, ff(96)),
               latent(20, 80, 32, 16, 40, 192, 0.11, 300.0)], width=192, vocab=259, scale=1.0)
# one head everywhere, wide heads, eps large enough to matter
WIDE = config([latent(1, 128, 64, 128, 128, 256, 0.07, 2e3), delta(1, 136, ff(72)), delta(1, 256)], width=128, vocab=77, scale=3.0,
              eps=1e-2)
# only one kind of mixer
ONLY_DELTA = config([delta(4, 16), delta(1, 96, ff(33))], width=64, vocab=50)
ONLY_LATENT = config([latent(4, 16, 16, 32, 24, 48, 0.3), latent(17, 16, 48, 48, 32, 64, 0.2, 50.0, ff(64))], width=64, vocab=50)

# several residual streams, differential attention: sizes that fit nothing; layers that read the cache of the first, with and
# without a layer between, with other constants; no feed-forward in places, at the end too
DIFF_ODD = stream_config([attention(6, 3, 10, 28, 0.4, 0.3, 0.9, 7, ff(50)), attention(6, 3, 10, 28, 0.7, 0.6, 0.2, 11, None, 0),
                          attention(5, 5, 7, 9, 0.5, 0.2, 0.4, 1, ff(37)), attention(6, 3, 10, 28, 0.3, 0.1, 1.5, 40, None, 0)],
                         width=90, vocab=131, streams=3, eps=1e-3)
# sizes the tensor-core kernels take as they are
DIFF_EVEN = stream_config([attention(8, 2, 48, 80, 0.2, 0.4, 0.5, 32, ff(200)), attention(12, 1, 16, 32, 0.3, 0.8, 0.3, 50, ff(96)),
                           attention(8, 2, 48, 80, 0.15, 0.25, 1.0, 16, ff(72), 0), attention(12, 1, 16, 32, 0.3, 0.5, 0.7, 64, None, 1)],
                          width=192, vocab=259, streams=2)
# values wider than a tile of the flash kernel, more query heads to a key head than a block of rows, wide keys
DIFF_WIDE = stream_config([attention(2, 1, 128, 256, 0.07, 0.3, 0.5, 20, ff(72)), attention(20, 1, 32, 64, 0.2, 0.5, 0.4, 100),
                           attention(2, 1, 128, 256, 0.1, 0.6, 0.2, 9, None, 0), attention(3, 3, 24, 144, 0.2, 0.5, 0.4, 64, ff(40))],
                          width=136, vocab=77, streams=4, eps=1e-2)
# one stream, one head, values narrower than keys, no temperature to speak of
DIFF_ONE = stream_config([attention(1, 1, 64, 16, 0.125, 0.0, 0.0, 1000), attention(1, 1, 64, 16, 0.2, 0.9, 2.0, 3, ff(33), 0)], width=64, vocab=50,
                         streams=1, eps=1e-1)

CONFIGS = {"odd": ODD, "even": EVEN, "wide": WIDE, "only_delta": ONLY_DELTA, "only_latent": ONLY_LATENT,
           "diff_odd": DIFF_ODD, "diff_even": DIFF_EVEN, "diff_wide": DIFF_WIDE, "diff_one": DIFF_ONE}
RANKS = {"odd": 5, "even": 24, "wide": 16, "only_delta": 1, "only_latent": 8, "diff_odd": 0, "diff_even": 0, "diff_wide": 0, "diff_one": 0}


def weights(name, seed=3):
    """(torch bf16 tensors, the same as float64 arrays)"""
    from reimagined_b200.stack import synthetic_weights
    w = synthetic_weights(CONFIGS[name], seed, RANKS[name])
    return w, {k: v.float().numpy().astype(np.float64) for k, v in w.items()}


def engine(name, dtype="float32", slots=3, capacity=400, seed=3, **kw):
    from reimagined_b200.stack import StackEngine
    w, p = weights(name, seed)
    return StackEngine(CONFIGS[name], w, dtype, slots, capacity, **kw), p


def tokens(name, n, seed=0):
    return np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], n).tolist()


def oracle_logits(name, params, ids):
    from oracle.layer_stack import decoder
    return decoder(CONFIGS[name], params).feed(ids)


# largest error of a row of logits, as a fraction of the logits' spread: fp32 rounding, and bf16 operands
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}


def row_errors(got, want):
    got = got.detach().cpu().numpy().astype(np.float64) if hasattr(got, "detach") else np.asarray(got, np.float64)
    return np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.std(want)


def close(got, want, dtype="float32"):
    e = row_errors(got, want)
    assert np.isfinite(e).all() and e.max() <= LIMIT[dtype], f"row {int(e.argmax())} of {len(e)}: {e.max():.3g}"
