"""Time the layer-stack operators and models, each beside the like operator of the ternary hybrid at the same size.

    python -m reimagined_b200.stack_shapes --width 4096 [--only dense,delta,latent,attention,norm,model] [--model guselix,goguvik]

One JSON line per record.  Every operator runs from a CUDA graph over several copies of its weights, states or caches, so
that a call never finds them in L2.  `roofline` is the share of min(bytes / copy bandwidth, FLOPs / bf16 GEMM rate) that
the call reaches; bytes and FLOPs are the algorithmic ones.
"""
from __future__ import annotations

import argparse
import ctypes as C
import json
import os
from typing import Callable, List, Optional

import torch

from . import capi

HBM_GBS, BF16_TFLOPS, INT8_TOPS, FP32_TFLOPS = 6650.0, 1590.0, 4500.0, 74.0


def use_measured_peaks() -> None:
    global HBM_GBS, BF16_TFLOPS
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            peaks = json.load(f)
        HBM_GBS, BF16_TFLOPS = peaks["hbm_gbs"], peaks["bf16_tflops"]


def stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def time_calls(calls: List[Callable], n: int = 20) -> float:
    """Microseconds per call, the calls in turn from one graph, best of three replays."""
    for f in calls[:3]:
        f()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(n):
            calls[i % len(calls)]()
    graph.replay()
    best = float("inf")
    for _ in range(3):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        best = min(best, a.elapsed_time(b) * 1e3 / n)
    return best


def record(op: str, us: float, nbytes: float, flops: float = 0.0, rate: Optional[float] = None, **more) -> dict:
    ideal = max(nbytes / HBM_GBS / 1e3, flops / (rate or BF16_TFLOPS) / 1e6)
    return {"op": op, **more, "us": round(us, 2), "gbs": round(nbytes / us / 1e3, 1), "tflops": round(flops / us / 1e6, 1),
            "roofline": round(ideal / us, 3)}


def copies(nbytes: float, most: int = 24) -> int:
    return max(1, min(most, int(300e6 / nbytes)))


def bf16(*shape, scale=0.02):
    return (torch.randn(*shape, device="cuda") * scale).bfloat16()


def check(rc: int, what: str) -> None:
    capi.check(rc, what, capi.stack_lib())


# ---- linear layers ------------------------------------------------------------------------------------------------------
def dense(m: int, k: int, n: int, residual: bool = False) -> dict:
    L = capi.stack_lib()
    ws = [bf16(n, k) for _ in range(copies(2.0 * n * k))]
    x, out = bf16(m, k, scale=1.0), torch.zeros(m, n, device="cuda")
    views = [capi.DenseView(w.data_ptr(), None, k, n) for w in ws]
    us = time_calls([lambda v=v: check(L.tbl_dense_forward(C.byref(v), capi.BF16, 0, x.data_ptr(), k, m, out.data_ptr() if residual else None,
                                                           out.data_ptr(), stream()), "tbl_dense_forward") for v in views])
    return record("dense + residual" if residual else "dense", us, 2.0 * (n * k + m * k) + 4.0 * m * n * (2 if residual else 1), 2.0 * m * n * k,
                  rows=m, k=k, n=n)


def gated(m: int, k: int, ff: int, activation: int = capi.ACT_SILU) -> dict:
    L = capi.stack_lib()
    ws = [bf16(2 * ff, k) for _ in range(copies(4.0 * ff * k))]
    x, out, bias = bf16(m, k, scale=1.0), torch.empty(m, ff, device="cuda", dtype=torch.bfloat16), torch.zeros(2 * ff, device="cuda")
    views = [capi.DenseView(w.data_ptr(), bias.data_ptr(), k, 2 * ff) for w in ws]
    us = time_calls([lambda v=v: check(L.tbl_gated_dense_act_forward(C.byref(v), capi.BF16, 0, activation, x.data_ptr(), k, m, ff, out.data_ptr(), stream()),
                                       "tbl_gated_dense_act_forward") for v in views])
    return record("gated dense, gelu" if activation == capi.ACT_GELU_TANH else "gated dense", us, 2.0 * (2 * ff * k + m * k + m * ff), 4.0 * m * ff * k, rows=m, k=k, n=ff)


def ternary(m: int, k: int, n: int) -> dict:
    """The hybrid's linear layer at the same size (2-bit weights, int8 activations, fp32 out)."""
    L = capi.lib()
    weights = []
    for _ in range(copies(n * k * (0.25 if m <= 64 else 1.0))):
        words = torch.randint(0, 2 ** 31 - 1, (n * k // 16,), dtype=torch.int32, device="cuda") & 0x2AAAAAAA
        strips = torch.empty(max(16, L.tbl_strip_bytes(n, k)), dtype=torch.uint8, device="cuda")
        capi.check(L.tbl_relayout_strips(words.data_ptr(), n, k, strips.data_ptr(), stream()), "tbl_relayout_strips")
        w8 = None
        if m > 64:
            w8 = torch.empty(n * k, dtype=torch.int8, device="cuda")
            capi.check(L.tbl_expand_weights_i8(words.data_ptr(), n, k, w8.data_ptr(), stream()), "tbl_expand_weights_i8")
        weights.append((words, strips, w8))
    x, y = torch.randn(m, k, device="cuda"), torch.empty(m, n, device="cuda")
    size = L.tbl_linear_workspace_bytes(m, k, n)
    ws = torch.empty(size, dtype=torch.uint8, device="cuda")
    us = time_calls([lambda w=w: capi.check(L.tbl_linear_forward(
        x.data_ptr(), w[0].data_ptr(), w[1].data_ptr(), w[2].data_ptr() if w[2] is not None else None, 0.02, m, k, n, 8, 0, None, None, y.data_ptr(),
        ws.data_ptr(), size, stream()), "tbl_linear_forward") for w in weights])
    return record("hybrid: ternary linear", us, n * k * (0.25 if m <= 64 else 1.0) + 4.0 * m * (k + n), 2.0 * m * n * k, INT8_TOPS, rows=m, k=k, n=n)


# ---- recurrences ----------------------------------------------------------------------------------------------------------
def delta(n_seq: int, n_tok: int, heads: int, dim: int, rank: int) -> dict:
    from .stack import DECAY_RATE, KEY_EPS
    L, hd, rows = capi.stack_lib(), heads * dim, n_seq * n_tok
    cols = 5 * hd + rank
    some, f32 = bf16(1, 8), torch.zeros(cols, device="cuda")
    w2, norm = bf16(hd, rank), torch.ones(hd, device="cuda")
    m = capi.DeltaMixer()
    m.in_, m.out = capi.DenseView(some.data_ptr(), f32.data_ptr(), 8, cols), capi.DenseView(some.data_ptr(), None, hd, 8)
    m.decay_up, m.norm = capi.DenseView(w2.data_ptr(), f32.data_ptr(), rank, hd), norm.data_ptr()
    m.heads, m.dim, m.rank, m.decay_rate, m.key_eps = heads, dim, rank, DECAY_RATE, KEY_EPS
    state = 4.0 * n_seq * hd * dim
    states = [torch.zeros(n_seq, heads, dim, dim, device="cuda") for _ in range(copies(state, 16) if n_tok == 1 else 1)]
    proj, out = torch.randn(rows, cols, device="cuda"), torch.empty(rows, hd, device="cuda", dtype=torch.bfloat16)
    slots = torch.arange(n_seq, dtype=torch.int32, device="cuda")
    size = L.tbl_delta_workspace_bytes(C.byref(m), capi.BF16, rows)
    ws = torch.empty(size, dtype=torch.uint8, device="cuda")
    us = time_calls([lambda s=s: check(L.tbl_delta_forward(C.byref(m), capi.BF16, 0, 1e-6, proj.data_ptr(), s.data_ptr(), slots.data_ptr(), n_seq, n_tok,
                                                           out.data_ptr(), ws.data_ptr(), size, stream()), "tbl_delta_forward") for s in states],
                    20 if n_tok == 1 else 4)
    # five multiply-adds per state element and token
    return record("delta rule", us, 2 * state + 4.0 * rows * cols + 2.0 * rows * hd, 10.0 * rows * hd * dim, FP32_TFLOPS, sequences=n_seq, tokens=n_tok,
                  heads=heads, dim=dim)


def ssd(n_seq: int, heads: int, d_head: int, d_state: int) -> dict:
    """The hybrid's recurrence for one token."""
    L, inner = capi.lib(), heads * d_head
    state = 4.0 * n_seq * inner * d_state
    xbc, dt = torch.randn(n_seq, inner + 2 * d_state, device="cuda"), torch.randn(n_seq, heads, device="cuda")
    a, y = torch.ones(heads, device="cuda"), torch.empty(n_seq, inner, device="cuda")
    states = [torch.zeros(n_seq, inner, d_state, device="cuda") for _ in range(copies(state, 16))]
    us = time_calls([lambda s=s: capi.check(L.tbl_mamba_ssd_step(xbc.data_ptr(), dt.data_ptr(), a.data_ptr(), a.data_ptr(), s.data_ptr(), y.data_ptr(),
                                                                 heads, d_head, d_state, 1, n_seq, stream()), "tbl_mamba_ssd_step") for s in states])
    return record("hybrid: SSD step", us, 2 * state + 8.0 * n_seq * inner, 5.0 * n_seq * inner * d_state, FP32_TFLOPS, sequences=n_seq, tokens=1,
                  heads=heads, dim=d_head, d_state=d_state)


# ---- attention ---------------------------------------------------------------------------------------------------------------
def latent(n_seq: int, n_tok: int, context: int, heads: int, dim: int = 128, rot: int = 64, vdim: int = 128, q_rank: int = 1536,
           kv_rank: int = 512) -> dict:
    """The whole mixer between its stacked projection and W_o: norms, W_uq, absorbed or expanded keys, attention, W_uv, gate."""
    L, rows = capi.stack_lib(), n_seq * n_tok
    cols = q_rank + kv_rank + rot + heads * vdim
    some, ones = bf16(1, 8), torch.ones(max(q_rank, kv_rank), device="cuda")
    uq, uk, ukt, uv = bf16(heads * (dim + rot), q_rank), bf16(heads * dim, kv_rank), bf16(heads * kv_rank, dim), bf16(heads * vdim, kv_rank)
    m = capi.LatentMixer()
    m.in_, m.out = capi.DenseView(some.data_ptr(), None, 8, cols), capi.DenseView(some.data_ptr(), None, heads * vdim, 8)
    m.uq, m.uk, m.uv = (capi.DenseView(w.data_ptr(), None, w.shape[1], w.shape[0]) for w in (uq, uk, uv))
    m.uk_t, m.q_norm, m.kv_norm = ukt.data_ptr(), ones.data_ptr(), ones.data_ptr()
    table = torch.ones(context, rot // 2, device="cuda")
    m.rope_cos, m.rope_sin, m.rope_positions = table.data_ptr(), table.data_ptr(), context
    m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale = heads, dim, rot, vdim, q_rank, kv_rank, (dim + rot) ** -0.5
    cache = 2.0 * n_seq * context * (kv_rank + rot)
    caches = [bf16(n_seq, context, kv_rank + rot, scale=1.0) for _ in range(copies(cache, 8) if n_tok == 1 else 1)]
    pos = torch.full((n_seq,), context - n_tok, dtype=torch.int32, device="cuda")
    slots = torch.arange(n_seq, dtype=torch.int32, device="cuda")
    proj, out = torch.randn(rows, cols, device="cuda"), torch.empty(rows, heads * vdim, device="cuda", dtype=torch.bfloat16)
    size = L.tbl_latent_workspace_bytes(C.byref(m), capi.BF16, n_seq, n_tok, context)
    ws = torch.empty(size, dtype=torch.uint8, device="cuda")
    us = time_calls([lambda c=c: check(L.tbl_latent_forward(C.byref(m), capi.BF16, 0, 1e-6, proj.data_ptr(), c.data_ptr(), context, slots.data_ptr(),
                                                            pos.data_ptr(), n_seq, n_tok, context, out.data_ptr(), ws.data_ptr(), size, stream()),
                                       "tbl_latent_forward") for c in caches], 16 if n_tok == 1 else 4)
    weights = 2.0 * (uq.numel() + uk.numel() + uv.numel())
    pairs = n_seq * sum(range(context - n_tok + 1, context + 1))
    project = 2.0 * rows * uq.numel()
    if n_tok == 1:           # in the latent space
        flops = project + 2.0 * rows * (uk.numel() + uv.numel()) + 2.0 * heads * pairs * (2 * kv_rank + rot)
    else:                    # keys and values expanded
        flops = project + 2.0 * n_seq * context * (uk.numel() + uv.numel()) + 2.0 * heads * pairs * (dim + rot + vdim)
    return record("latent attention", us, cache + weights + 4.0 * rows * cols, flops, sequences=n_seq, tokens=n_tok, context=context, heads=heads)


def differential(n_seq: int, n_tok: int, context: int, heads: int, kv_heads: int, dim: int = 64, vdim: int = 128, maps: int = 2) -> dict:
    """The whole mixer between its stacked projection and W_o: cache append, attention, combination of the maps, head norm, gate."""
    L, rows = capi.stack_lib(), n_seq * n_tok
    cols = heads * (maps * dim + vdim) + kv_heads * (maps * dim + vdim)
    some, zeros = bf16(1, 8), torch.zeros(cols, device="cuda")
    m = capi.AttentionMixer()
    m.in_, m.out = capi.DenseView(some.data_ptr(), zeros.data_ptr(), 8, cols), capi.DenseView(some.data_ptr(), None, heads * vdim, 8)
    table = torch.ones(context, device="cuda")
    m.temperature, m.temperature_positions, m.heads, m.kv_heads, m.dim, m.vdim, m.maps, m.gated = table.data_ptr(), context, heads, kv_heads, dim, vdim, maps, 1
    m.kv_from, m.scale, m.lambda_, m.out_scale = -1, dim ** -0.5, 0.5, 0.5
    per_token = kv_heads * L.tbl_attention_cache_width(C.byref(m))
    cache = 2.0 * n_seq * context * per_token
    caches = [bf16(n_seq, context * per_token, scale=1.0) for _ in range(copies(cache, 16) if n_tok == 1 else 1)]
    pos = torch.full((n_seq,), context - n_tok, dtype=torch.int32, device="cuda")
    slots = torch.arange(n_seq, dtype=torch.int32, device="cuda")
    proj, out = torch.randn(rows, cols, device="cuda"), torch.empty(rows, heads * vdim, device="cuda", dtype=torch.bfloat16)
    size = L.tbl_attention_workspace_bytes(C.byref(m), capi.BF16, n_seq, n_tok, context)
    ws = torch.empty(size, dtype=torch.uint8, device="cuda")
    us = time_calls([lambda c=c: check(L.tbl_attention_forward(C.byref(m), capi.BF16, 0, 1e-6, proj.data_ptr(), c.data_ptr(), n_seq, context, slots.data_ptr(),
                                                               pos.data_ptr(), n_seq, n_tok, context, out.data_ptr(), ws.data_ptr(), size, stream()),
                                       "tbl_attention_forward") for c in caches], 16 if n_tok <= 8 else 4)
    pairs = n_seq * sum(range(context - n_tok + 1, context + 1))
    name = "differential attention" if maps == 2 else "attention"
    return record(name, us, cache + 4.0 * rows * cols + 2.0 * rows * heads * vdim, 2.0 * heads * maps * pairs * (dim + vdim), sequences=n_seq, tokens=n_tok,
                  context=context, heads=heads, kv_heads=kv_heads)


def attention(n_seq: int, context: int, heads: int, dim: int) -> dict:
    """The hybrid's attention for one token (its kernel's shared memory bounds the context)."""
    L, kv = capi.lib(), heads * dim
    cache = 8.0 * n_seq * context * kv
    pairs = [(torch.randn(n_seq, context, kv, device="cuda"), torch.randn(n_seq, context, kv, device="cuda")) for _ in range(copies(cache, 8))]
    q, new, out = torch.randn(n_seq, kv, device="cuda"), torch.randn(n_seq, 2 * kv, device="cuda"), torch.empty(n_seq, kv, device="cuda")
    table = torch.ones(context, dim // 2, device="cuda")
    pos = torch.full((n_seq,), context - 1, dtype=torch.int32, device="cuda")
    us = time_calls([lambda c=c: capi.check(L.tbl_attention_decode(q.data_ptr(), new.data_ptr(), c[0].data_ptr(), c[1].data_ptr(), context, pos.data_ptr(),
                                                                   table.data_ptr(), table.data_ptr(), context, heads, heads, dim, context, n_seq,
                                                                   out.data_ptr(), stream()), "tbl_attention_decode") for c in pairs], 16)
    return record("hybrid: attention step", us, cache, 4.0 * n_seq * context * kv, FP32_TFLOPS, sequences=n_seq, tokens=1, context=context, heads=heads)


# ---- norms --------------------------------------------------------------------------------------------------------------------
def depth(rows: int, width: int, count: int) -> dict:
    L = capi.stack_lib()
    h = [torch.randn(count, rows, width, device="cuda") for _ in range(copies(4.0 * count * rows * width, 8))]
    w, norm = torch.randn(count, device="cuda"), torch.ones(width, device="cuda")
    x, out = torch.empty(rows, width, device="cuda"), torch.empty(rows, width, device="cuda", dtype=torch.bfloat16)
    us = time_calls([lambda a=a: check(L.tbl_depth_norm(a.data_ptr(), rows * width, count, w.data_ptr(), capi.BF16, None, rows, width, 1e-6,
                                                        norm.data_ptr(), x.data_ptr(), out.data_ptr(), stream()), "tbl_depth_norm") for a in h])
    return record("depth average + norm", us, rows * width * (4.0 * count + 6), rows=rows, width=width, arrays=count)


def streams(rows: int, width: int, count: int) -> dict:
    """A boundary between sublayers: the streams updated in place, the next input, Dynamic Tanh."""
    L = capi.stack_lib()
    xs = [torch.randn(count, rows, width, device="cuda") for _ in range(copies(4.0 * count * rows * width, 8))]
    y, norm = torch.randn(rows, width, device="cuda"), torch.ones(width, device="cuda")
    mix, w = torch.eye(count, device="cuda"), torch.ones(count, device="cuda")
    out = torch.empty(rows, width, device="cuda", dtype=torch.bfloat16)
    us = time_calls([lambda a=a: check(L.tbl_stream_norm(a.data_ptr(), rows * width, count, y.data_ptr(), mix.data_ptr(), w.data_ptr(), 1, w.data_ptr(),
                                                         capi.BF16, None, rows, width, capi.NORM_DYNAMIC_TANH, 1e-6, 0.5, norm.data_ptr(), norm.data_ptr(),
                                                         None, out.data_ptr(), stream()), "tbl_stream_norm") for a in xs])
    return record("stream update + norm", us, rows * width * (8.0 * count + 6), rows=rows, width=width, streams=count)


def row_norm(rows: int, width: int) -> dict:
    L = capi.lib()
    xs = [torch.randn(rows, width, device="cuda") for _ in range(copies(4.0 * rows * width, 8))]
    w, out = torch.ones(width, device="cuda"), torch.empty(rows, width, device="cuda")
    us = time_calls([lambda a=a: capi.check(L.tbl_row_norm(a.data_ptr(), None, w.data_ptr(), rows, width, 1e-6, out.data_ptr(), 8, None, None, None,
                                                           stream()), "tbl_row_norm") for a in xs])
    return record("hybrid: row norm", us, rows * width * 8.0, rows=rows, width=width)


# ---- whole models ---------------------------------------------------------------------------------------------------------------
def guselix_config(width: int, layers: int, vocab: int = 32000) -> dict:
    """Sizes like a real model's: every fourth layer attends, every layer has a feed-forward; random weights."""
    heads, mlp = width // 128, {"kind": "dense", "ff": 3 * width}
    mix = {"type": "general_delta", "mixer": {"heads": heads, "dim": 128}, "mlp": mlp}
    att = {"type": "latent_attention", "mlp": mlp,
           "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 3 * width // 8, "kv_rank": 512, "scale": 192 ** -0.5,
                     "rot": {"base": 10000.0, "dims": 64}}}
    return {"architecture": "Guselix", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "vocab": vocab, "width": width,
            "layers": [att if i % 4 == 3 else mix for i in range(layers)]}


def goguvik_config(width: int, layers: int, vocab: int = 32000) -> dict:
    """Sizes like a real model's: heads of two maps of 64 over values of 128, four query heads to a key/value head, every
    other layer over the cache of the one before it; random weights."""
    heads = width // 128
    out = []
    for i in range(layers):
        m = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 64, "vdim": 128, "scale": 0.125, "diff": 0.4, "q_temp": {"coef": 0.1, "every": 8192}}
        if i % 2:
            m["kv_from"] = i - 1
        out.append({"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": 3 * width}})
    return {"architecture": "Goguvik", "layers": out, "norm": {"eps": 1e-6}, "streams": 2, "vocab": vocab, "width": width}


CONFIGS = {"guselix": guselix_config, "goguvik": goguvik_config}


def time_stack(name: str, width: int, layers: int, batches=(1, 8, 64), context: int = 512, prompts=(512, 8192), iters: int = 50) -> List[dict]:
    from .stack import StackEngine, synthetic_weights
    cfg = CONFIGS[name](width, layers)
    weights = synthetic_weights(cfg, 1, rank=width // 32, device="cuda")
    params, out = sum(w.numel() for w in weights.values()), []
    for batch, prompt in [(b, 0) for b in batches] + [(1, p) for p in prompts]:
        eng = StackEngine(cfg, weights, slots=batch, capacity=max(prompt, context + iters + 8))
        slots = [eng.open() for _ in range(batch)]
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        rec = {"model": cfg["architecture"], "width": width, "layers": layers, "parameters": params}
        if prompt:
            ids, times = torch.randint(0, cfg["vocab"], (prompt,)).tolist(), []
            for _ in range(4):
                slot = eng.open() if eng._free else slots[0]
                a.record()
                eng.step([slot], [ids])
                b.record()
                torch.cuda.synchronize()
                times.append(a.elapsed_time(b))
                eng.close(slot)
            ms = min(times[1:])
            rec.update(phase="prefill", prompt=prompt, ms=round(ms, 3), tokens_per_s=round(prompt / ms * 1e3, 1))
        else:
            ids = torch.randint(0, cfg["vocab"], (batch, context)).tolist()
            for s, row in zip(slots, ids):
                eng.feed(s, row)
            tokens = [[row[0]] for row in ids]
            for _ in range(3):
                eng.step(slots, tokens)
            torch.cuda.synchronize()
            a.record()
            for _ in range(iters):
                eng.step(slots, tokens)
            b.record()
            torch.cuda.synchronize()
            us = a.elapsed_time(b) * 1e3 / iters
            rec.update(phase="decode", batch=batch, context=context, launches=eng.launches_per_step, us_per_step=round(us, 1),
                       tokens_per_s=round(batch / us * 1e6, 1),
                       weight_stream=round(2.0 * (params - weights["embed"].numel() + cfg["vocab"] * width) / us / 1e3 / HBM_GBS, 3))
        rec["device_status"] = eng.device_status()
        out.append(rec)
        del eng
        torch.cuda.empty_cache()
    return out


def time_hybrid(width: int, layers: int, batches=(1, 8, 64), context: int = 512, iters: int = 50) -> List[dict]:
    """The ternary hybrid at the same width and depth, every fourth block with attention; it has no prefill step."""
    from .decode import time_decode
    cfg = dict(num_layers=layers, d_model=width, vocab_size=32000, n_heads=width // 128, n_kv_heads=width // 128, mamba_d_state=16, mamba_expand=2,
               mamba_conv_kernel=4, mamba_head_dim=64, mamba_n_groups=1, attention_period=4, attention_slot=3)
    out = []
    for batch in batches:
        r = time_decode(batch, iters, context, cfg)
        out.append({"model": "JambaHybrid", "width": width, "layers": layers, "phase": "decode", "batch": batch, "context": context,
                    "launches": r["kernel_launches_per_step"], "us_per_step": r["us_per_step"], "tokens_per_s": r["tokens_per_s"],
                    "ternary_weights": r["ternary_weights"], "weight_stream": round(r["packed_mb"] * 1e6 / r["us_per_step"] / 1e3 / HBM_GBS, 3)})
        torch.cuda.empty_cache()
    return out


def operators(width: int, only=("dense", "delta", "latent", "attention", "norm")):
    """Generator of records at one model width."""
    heads, ff = width // 128, 3 * width
    if "dense" in only:
        for m in (1, 8, 64, 2048, 8192):
            yield dense(m, width, 5 * width + width // 32)
            yield ternary(m, width, 5 * width)
            yield dense(m, width, width, residual=True)
            yield ternary(m, width, width)
            yield gated(m, width, ff)
            yield gated(m, width, ff, capi.ACT_GELU_TANH)
            yield dense(m, ff, width, residual=True)
            yield ternary(m, ff, width)
    if "delta" in only:
        for n_seq in (1, 8, 64):
            yield delta(n_seq, 1, heads, 128, width // 32)
            yield ssd(n_seq, 2 * width // 64, 64, 16)
        for n_tok in (512, 8192):
            yield delta(1, n_tok, heads, 128, width // 32)
    if "latent" in only:
        for n_seq, context in ((1, 1024), (1, 8192), (8, 8192), (64, 4096)):
            yield latent(n_seq, 1, context, heads, q_rank=3 * width // 8)
            if n_seq <= 8:
                yield attention(n_seq, context, heads, 128)
        for n_tok in (512, 2048, 8192):
            yield latent(1, n_tok, n_tok, heads, q_rank=3 * width // 8)
    if "attention" in only:
        for n_seq, context in ((1, 1024), (1, 8192), (8, 8192), (64, 4096)):
            yield differential(n_seq, 1, context, heads, max(1, heads // 4))
            if n_seq <= 8 and "latent" not in only:
                yield attention(n_seq, context, heads, 128)
        for n_tok in (512, 2048, 8192):
            yield differential(1, n_tok, n_tok, heads, max(1, heads // 4))
    if "norm" in only:
        for rows in (1, 64, 8192):
            yield streams(rows, width, 2)
            yield streams(rows, width, 4)
            yield depth(rows, width, 9)
            yield row_norm(rows, width)


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--layers", type=int, default=4, help="layers of the whole-model timings")
    ap.add_argument("--only", default="dense,delta,latent,attention,norm,model")
    ap.add_argument("--model", default="guselix,goguvik", help="layer-stack models of the whole-model timings")
    args = ap.parse_args()
    use_measured_peaks()
    only = args.only.split(",")
    for r in operators(args.width, only):
        print(json.dumps(r), flush=True)
    if "model" in only:
        for name in args.model.split(","):
            for r in time_stack(name, args.width, args.layers):
                print(json.dumps(r), flush=True)
        for r in time_hybrid(args.width, args.layers):
            print(json.dumps(r), flush=True)


if __name__ == "__main__":
    main()
