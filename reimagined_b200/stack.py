"""Layer-stack models: decoder-only stacks of mixers with dense bfloat16 weights, served through `tbl_stack_step`.

A design is a list of layers in its configuration; every layer names its mixer and, optionally, a gated feed-forward:

    {"architecture": ..., "vocab": .., "width": .., "embedding": {"scale": ..}, "norm": {"eps": ..},
     "layers": [{"type": <mixer>, "mixer": {sizes and constants}, "mlp": {"kind": "dense", "ff": ..} or null}, ...]}

`MIXERS` maps a mixer's name to the code that says which tensors it has and how they become the library's descriptor,
and `DESIGNS` an architecture to what surrounds its mixers (norm, residual, feed-forward), so another design that uses the
same mechanisms in another order needs no new code.  `StackEngine` owns the device state of a number of sequences (slots)
and runs steps: portions of prompts and decode steps of several sequences, the latter replayed from CUDA graphs.  torch
owns device memory and streams only.

Guselix is this family with the mixers `general_delta` (delta rule with per-channel decay and removal rate) and
`latent_attention`, RMS norms and a learned average over the depth after every layer.  Goguvik has the mixer `attention`
(differential, grouped key/value heads, query temperature, layers that read an earlier layer's cache), Dynamic Tanh norms
and several residual streams ("streams") joined by hyper-connections.
"""
from __future__ import annotations

import ctypes as C
import math
import os
from typing import Callable, Dict, Iterable, List, NamedTuple, Optional, Sequence, Set, Tuple

import numpy as np
import torch

from . import capi
from .checkpoint import read_config, read_safetensors

Shapes = Dict[str, Tuple[int, ...]]

# constants of the delta rule that the design fixes
DECAY_RATE = math.exp(-0.5)       # decay = exp(-DECAY_RATE * sigmoid(.))
KEY_EPS = 1e-6                    # unit key: k / sqrt(sum k^2 + KEY_EPS)


class Mixer(NamedTuple):
    shapes: Callable              # (mixer config, width, rank of the low-rank decay) -> {suffix: shape}
    fill: Callable                # (engine, descriptor layer, prefix, mixer config) -> None


def _delta_shapes(m: dict, width: int, rank: int) -> Shapes:
    hd = m["heads"] * m["dim"]
    return {"r": (hd, width), "k": (hd, width), "v": (hd, width), "g": (hd, width), "a": (hd, width), "a.b": (hd,),
            "w1": (rank, width), "w2": (hd, rank), "w0": (hd,), "norm": (hd,), "o": (width, hd)}


def _fill_delta(e: "StackEngine", layer: capi.StackLayer, p: str, m: dict) -> None:
    d, hd = layer.delta, m["heads"] * m["dim"]
    layer.mixer = capi.MIXER_GENERAL_DELTA
    d.heads, d.dim, d.rank = m["heads"], m["dim"], e.weights[p + "w1"].shape[0]
    d.decay_rate, d.key_eps = DECAY_RATE, KEY_EPS
    bias = torch.zeros(5 * hd + d.rank)
    bias[4 * hd:5 * hd] = e.weights[p + "a.b"].float()
    d.in_ = e.dense([p + n for n in ("r", "k", "v", "g", "a", "w1")], bias)
    d.decay_up = e.dense([p + "w2"], e.weights[p + "w0"])
    d.out = e.dense([p + "o"])
    d.norm = e.f32(e.weights[p + "norm"])


def _latent_shapes(m: dict, width: int, rank: int) -> Shapes:
    h, d, rd, vd, q, r = (m[n] for n in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
    return {"dq": (q, width), "dq.norm": (q,), "uq": (h * (d + rd), q), "dkv": (r + rd, width), "dkv.norm": (r,),
            "uk": (h * d, r), "uv": (h * vd, r), "g": (h * vd, width), "o": (width, h * vd)}


def _fill_latent(e: "StackEngine", layer: capi.StackLayer, p: str, m: dict) -> None:
    a = layer.latent
    layer.mixer = capi.MIXER_LATENT_ATTENTION
    a.heads, a.dim, a.rot_dim, a.vdim = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    a.q_rank, a.kv_rank, a.scale = m["q_rank"], m["kv_rank"], float(m["scale"])
    if m["rot"]["dims"] != m["rot_dim"]:
        raise ValueError("latent_attention rotates all of its rotated part (rot.dims == rot_dim)")
    a.in_ = e.dense([p + n for n in ("dq", "dkv", "g")])
    a.uq, a.uk, a.uv, a.out = (e.dense([p + n]) for n in ("uq", "uk", "uv", "o"))
    uk = e.weights[p + "uk"].cuda().reshape(m["heads"], m["dim"], m["kv_rank"])
    a.uk_t = e._bf16(uk.transpose(1, 2)).data_ptr()
    a.q_norm, a.kv_norm = e.f32(e.weights[p + "dq.norm"]), e.f32(e.weights[p + "dkv.norm"])
    a.rope_positions = e.capacity
    a.rope_cos, a.rope_sin = e.rotation(float(m["rot"]["base"]), m["rot_dim"])


def _attention_shapes(m: dict, width: int, rank: int) -> Shapes:
    h, g, d, vd = (m[n] for n in ("heads", "kv_heads", "dim", "vdim"))
    rows = {"q": h * 2 * d}
    if m.get("kv_from") is None:
        rows.update(k=g * 2 * d, v=g * vd)
    out = {name: (n, width) for name, n in rows.items()}
    out.update({name + ".b": (n,) for name, n in rows.items()})
    out.update({name: (d,) for name in ("lq1", "lk1", "lq2", "lk2")})
    return {**out, "g": (h * vd, width), "o": (width, h * vd), "o.b": (width,)}


def _fill_attention(e: "StackEngine", layer: capi.StackLayer, p: str, m: dict) -> None:
    a, w, source = layer.attention, e.weights, m.get("kv_from")
    layer.mixer = capi.MIXER_ATTENTION
    a.heads, a.kv_heads, a.dim, a.vdim, a.maps, a.gated = m["heads"], m["kv_heads"], m["dim"], m["vdim"], 2, 1
    a.scale, a.kv_from = float(m["scale"]), -1 if source is None else source
    names = ["q"] if source is not None else ["q", "k", "v"]
    bias = torch.cat([w[p + n + ".b"].float() for n in names] + [w[p + "q.b"].new_zeros(m["heads"] * m["vdim"]).float()])
    a.in_ = e.dense([p + n for n in names + ["g"]], bias)
    a.out = e.dense([p + "o"], w[p + "o.b"])
    dot = lambda x, y: float((w[p + x].double() * w[p + y].double()).sum())
    a.lambda_ = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + float(m["diff"])
    a.out_scale = 1.0 - float(m["diff"])
    if m.get("q_temp") is not None:
        a.temperature, a.temperature_positions = e.query_temperature(float(m["q_temp"]["coef"]), m["q_temp"]["every"]), e.capacity


MIXERS: Dict[str, Mixer] = {
    "general_delta": Mixer(_delta_shapes, _fill_delta),
    "latent_attention": Mixer(_latent_shapes, _fill_latent),
    "attention": Mixer(_attention_shapes, _fill_attention),
}


class Design(NamedTuple):
    """What an architecture fixes around its mixers."""
    norm: int                     # capi.NORM_*
    activation: int               # capi.ACT_* of the feed-forward
    ff_bias: bool
    depth_average: bool           # learned average over the depth after every layer
    streams: bool                 # several residual streams with hyper-connections; their number is in the configuration


DESIGNS: Dict[str, Design] = {
    "Guselix": Design(capi.NORM_RMS, capi.ACT_SILU, ff_bias=True, depth_average=True, streams=False),
    "Goguvik": Design(capi.NORM_DYNAMIC_TANH, capi.ACT_GELU_TANH, ff_bias=False, depth_average=False, streams=True),
}


def design_of(cfg: dict) -> Design:
    if cfg["architecture"] not in DESIGNS:
        raise ValueError(f"no layer-stack design named {cfg['architecture']!r}")
    return DESIGNS[cfg["architecture"]]


def _sublayer_shapes(design: Design, cfg: dict, p: str, n: int) -> Shapes:
    """The tensors around sublayer n (1: mixer, 2: feed-forward) of a layer."""
    out = _norm_shapes(design, f"{p}norm{n}", cfg["width"])
    if design.streams:
        s = cfg["streams"]
        out.update({f"{p}hc{n}.in": (s,), f"{p}hc{n}.out": (s,), f"{p}hc{n}.mix": (s, s)})
    return out


def _norm_shapes(design: Design, name: str, width: int) -> Shapes:
    out = {name: (width,)}
    if design.norm == capi.NORM_DYNAMIC_TANH:
        out.update({name + ".b": (width,), name + ".alpha": ()})
    return out


def tensor_shapes(cfg: dict, ranks: Sequence[int]) -> Shapes:
    """Every tensor of a configuration; ranks[i] is the rank of layer i's low-rank decay (it is not in the
    configuration: the tensor's shape gives it)."""
    design, width = design_of(cfg), cfg["width"]
    out = {"embed": (cfg["vocab"], width), **_norm_shapes(design, "final.norm", width)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] not in MIXERS:
            raise ValueError(f"layer {i}: no mixer named {layer['type']!r}")
        out.update(_sublayer_shapes(design, cfg, p, 1))
        for name, shape in MIXERS[layer["type"]].shapes(layer["mixer"], width, ranks[i]).items():
            out[p + "mix." + name] = shape
        if layer["mlp"] is not None:
            if layer["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: no feed-forward of the kind {layer['mlp']['kind']!r}")
            ff = layer["mlp"]["ff"]
            out.update(_sublayer_shapes(design, cfg, p, 2))
            for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
                out[p + "mlp." + name] = shape
                if design.ff_bias:
                    out[p + "mlp." + name + ".b"] = shape[:1]
        if design.depth_average:
            out[p + "dwa"] = (i + 2,)
    return out


def _unused_tensors(cfg: dict) -> Set[str]:
    """Tensors that a checkpoint may hold although nothing reads them: around the feed-forward a layer does not have."""
    design = design_of(cfg)
    return {name for i, layer in enumerate(cfg["layers"]) if layer["mlp"] is None for name in _sublayer_shapes(design, cfg, f"l{i}.", 2)}


def check_weights(cfg: dict, weights: Dict[str, torch.Tensor]) -> None:
    ranks = [weights[f"l{i}.mix.w1"].shape[0] if f"l{i}.mix.w1" in weights else 0 for i in range(len(cfg["layers"]))]
    want = tensor_shapes(cfg, ranks)
    missing, extra = sorted(set(want) - set(weights)), sorted(set(weights) - set(want) - _unused_tensors(cfg))
    if missing or extra:
        raise ValueError(f"weights do not fit the configuration: missing {missing[:5]}, unknown {extra[:5]}")
    for name, shape in want.items():
        if tuple(weights[name].shape) != tuple(shape):
            raise ValueError(f"{name} has the shape {tuple(weights[name].shape)}, expected {tuple(shape)}")


def synthetic_weights(cfg: dict, seed: int = 1, rank: int = 16, device: str = "cpu") -> Dict[str, torch.Tensor]:
    """Random weights of a configuration, scaled so that activations stay of order one."""
    gen = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, [rank] * len(cfg["layers"])).items():
        w = torch.randn(shape, generator=gen, device=device)
        if name.endswith("dwa"):
            w = 0.1 * w
            w[-1] += 1.0
        elif ".hc" in name:
            w = 0.2 * w + (torch.eye(shape[0], device=device) if name.endswith(".mix") else 1.0 / shape[0] if name.endswith(".in") else 1.0)
        elif name.endswith(".alpha"):
            w = 0.5 + 0.1 * w.clamp(-3.0, 3.0)
        elif name.endswith(".b"):
            w = 0.1 * w
        elif ".mix.l" in name:
            w = 0.5 * shape[0] ** -0.5 * w
        elif name.endswith("norm") or ".norm" in name:
            w = 1.0 + 0.1 * w
        elif len(shape) == 2 and name != "embed":
            w = w * shape[1] ** -0.5
        elif len(shape) == 1:
            w = 0.1 * w
        out[name] = w.to(torch.bfloat16)
    return out


class StackEngine:
    """Device state of `slots` sequences of up to `capacity` tokens, and the steps that advance them."""

    PORTION = 8192                # most rows of one step; longer prompts are fed in portions
    MAX_GRAPHS = 32

    def __init__(self, cfg: dict, weights: Dict[str, torch.Tensor], dtype: str = "bfloat16", slots: int = 1,
                 capacity: int = 1024, graphs: bool = True):
        if not torch.cuda.is_available():
            raise RuntimeError("layer-stack models run on CUDA devices only (no CPU fallback)")
        check_weights(cfg, weights)
        self.L = capi.stack_lib()
        self.cfg, self.weights, self.design = cfg, weights, design_of(cfg)
        self.precision = {"float32": capi.F32, "bfloat16": capi.BF16}[dtype]
        self.slots, self.capacity, self.graphs = int(slots), int(capacity), graphs
        self.vocab, self.width, self.n_layers = cfg["vocab"], cfg["width"], len(cfg["layers"])
        self._keep: List[torch.Tensor] = []
        self._rotations: Dict[Tuple[float, int], Tuple[int, int]] = {}
        self._temperatures: Dict[tuple, int] = {}
        self._build()
        del self.weights
        m = C.byref(self.model)
        nbytes = self.L.tbl_stack_state_bytes(m, self.precision, self.slots, self.capacity)
        if nbytes == 0:
            raise ValueError("the library rejected the model description (sizes out of range)")
        self.state = torch.empty(nbytes, dtype=torch.uint8, device="cuda")
        self.workspace = torch.empty(0, dtype=torch.uint8, device="cuda")
        self.length = [0] * self.slots
        self._free = list(range(self.slots))
        self._graphs: Dict[Tuple[int, int], tuple] = {}
        self._reset(-1)
        self.device_status()      # one-time library state is set up before anything is captured

    # ---- weights ------------------------------------------------------------------------------------------------
    def f32(self, t: torch.Tensor) -> int:
        t = t.to(device="cuda", dtype=torch.float32).contiguous()
        self._keep.append(t)
        return t.data_ptr()

    def _bf16(self, t: torch.Tensor) -> torch.Tensor:
        t = t.to(device="cuda", dtype=torch.bfloat16).contiguous()
        self._keep.append(t)
        return t

    def dense(self, names: Iterable[str], bias: Optional[torch.Tensor] = None) -> capi.DenseView:
        """The rows of the named tensors stacked in one linear layer."""
        w = self._bf16(torch.cat([self.weights[n].cuda() for n in names]))
        return capi.DenseView(w.data_ptr(), None if bias is None else self.f32(bias), w.shape[1], w.shape[0])

    def rotation(self, base: float, dims: int) -> Tuple[int, int]:
        """cos / sin of position * base^(-2i/dims), worked out in double precision."""
        if (base, dims) not in self._rotations:
            freq = base ** (-2.0 * np.arange(dims // 2) / dims)
            ang = np.arange(self.capacity, dtype=np.float64)[:, None] * freq[None, :]
            self._rotations[base, dims] = self.f32(torch.from_numpy(np.cos(ang))), self.f32(torch.from_numpy(np.sin(ang)))
        return self._rotations[base, dims]

    def query_temperature(self, coef: float, every) -> int:
        """1 + coef * ln(floor((position + 1) / every) + 1), worked out in double precision."""
        if (coef, every) not in self._temperatures:
            steps = np.floor_divide(np.arange(1, self.capacity + 1), every)
            self._temperatures[coef, every] = self.f32(torch.from_numpy(1.0 + coef * np.log(steps + 1.0)))
        return self._temperatures[coef, every]

    def norm(self, name: str) -> Tuple[int, capi.TanhNorm]:
        """A norm's weight, and what Dynamic Tanh has beside it."""
        extra = capi.TanhNorm()
        if self.design.norm == capi.NORM_DYNAMIC_TANH:
            extra.bias, extra.alpha = self.f32(self.weights[name + ".b"]), float(self.weights[name + ".alpha"])
        return self.f32(self.weights[name]), extra

    def hyper(self, prefix: str) -> capi.Hyper:
        if not self.design.streams:
            return capi.Hyper()
        return capi.Hyper(*(self.f32(self.weights[prefix + n]) for n in ("in", "mix", "out")))

    def _paired(self, gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
        """Gate and up rows in alternating blocks, the last block filled with zero rows."""
        b = capi.PAIR_BLOCK
        pad = (-gate.shape[0]) % b
        both = []
        for t in (gate, up):
            t = t.cuda()
            t = torch.cat([t, t.new_zeros((pad,) + tuple(t.shape[1:]))])
            both.append(t.reshape((-1, 1, b) + tuple(t.shape[1:])))
        return torch.cat(both, dim=1).flatten(0, 2)

    def _build(self) -> None:
        cfg, w = self.cfg, self.weights
        self._layers = (capi.StackLayer * self.n_layers)()
        for i, c in enumerate(cfg["layers"]):
            layer, p = self._layers[i], f"l{i}."
            layer.norm1, layer.tanh1 = self.norm(p + "norm1")
            layer.hyper1 = self.hyper(p + "hc1.")
            MIXERS[c["type"]].fill(self, layer, p + "mix.", c["mixer"])
            if c["mlp"] is not None:
                layer.ff, layer.activation = c["mlp"]["ff"], self.design.activation
                layer.norm2, layer.tanh2 = self.norm(p + "norm2")
                layer.hyper2 = self.hyper(p + "hc2.")
                gu = self._bf16(self._paired(w[p + "mlp.gate"], w[p + "mlp.up"]))
                bias = self.f32(self._paired(w[p + "mlp.gate.b"], w[p + "mlp.up.b"])) if self.design.ff_bias else None
                layer.gate_up = capi.DenseView(gu.data_ptr(), bias, gu.shape[1], gu.shape[0])
                layer.down = self.dense([p + "mlp.down"], w[p + "mlp.down.b"] if self.design.ff_bias else None)
            if self.design.depth_average:
                layer.depth_weights = self.f32(w[p + "dwa"])
        model = capi.StackModel()
        model.width, model.vocab, model.n_layers = self.width, self.vocab, self.n_layers
        embed = self._bf16(w["embed"])
        model.embedding, model.embedding_scale = embed.data_ptr(), float(cfg.get("embedding", {}).get("scale", 1.0))
        model.norm_kind, model.norm_eps = self.design.norm, float(cfg["norm"]["eps"])
        model.streams = cfg["streams"] if self.design.streams else 0
        model.layers = C.cast(self._layers, C.POINTER(capi.StackLayer))
        model.final_norm, model.final_tanh = self.norm("final.norm")
        model.head = capi.DenseView(embed.data_ptr(), None, self.width, self.vocab)
        self.model = model

    # ---- sequences -----------------------------------------------------------------------------------------------
    def _stream(self) -> int:
        return torch.cuda.current_stream().cuda_stream

    def _reset(self, slot: int) -> None:
        capi.check(self.L.tbl_stack_state_reset(C.byref(self.model), self.precision, self.slots, self.capacity, slot,
                                                self.state.data_ptr(), self.state.numel(), self._stream()),
                   "tbl_stack_state_reset", self.L)

    def open(self) -> int:
        """A slot with an empty sequence."""
        if not self._free:
            raise RuntimeError("every slot is in use")
        slot = self._free.pop(0)
        self._reset(slot)
        self.length[slot] = 0
        return slot

    def close(self, slot: int) -> None:
        if slot in self._free or not 0 <= slot < self.slots:
            raise ValueError(f"slot {slot} is not open")
        self._free.append(slot)

    # ---- steps -----------------------------------------------------------------------------------------------------
    def _enqueue(self, slots, n_seq, n_tok, context, tokens, want, n_want, logits, trace, workspace) -> None:
        capi.check(self.L.tbl_stack_step(
            C.byref(self.model), self.precision, self.slots, self.capacity, self.state.data_ptr(), slots.data_ptr(), n_seq,
            n_tok, context, tokens.data_ptr(), None if n_want == 0 else want.data_ptr(), n_want,
            None if n_want == 0 else logits.data_ptr(), None if trace is None else trace.data_ptr(), workspace.data_ptr(),
            workspace.numel(), self._stream()), "tbl_stack_step", self.L)

    def _workspace_bytes(self, n_seq: int, n_tok: int, context: int) -> int:
        return self.L.tbl_stack_workspace_bytes(C.byref(self.model), self.precision, n_seq, n_tok, context)

    def step(self, slots: Sequence[int], tokens, want: Optional[Sequence[int]] = None, trace: bool = False):
        """One step: tokens [len(slots)][n] (the same n for every sequence) -> logits fp32 [len(want), vocab] of the
        wanted rows (row = sequence * n + token; default: the last token of every sequence).  With `trace` also the
        residual stream after every layer, [layers, rows, width]."""
        ids = torch.as_tensor(tokens, dtype=torch.int32).reshape(len(slots), -1)
        n_seq, n_tok = ids.shape
        if n_tok == 0 or len(set(slots)) != n_seq or any(s in self._free or not 0 <= s < self.slots for s in slots):
            raise ValueError("a step needs distinct open slots and at least one token each")
        if int(ids.min()) < 0 or int(ids.max()) >= self.vocab:
            raise ValueError("token id outside the vocabulary")
        longest = max(self.length[s] for s in slots) + n_tok
        if longest > self.capacity:
            raise ValueError(f"a sequence would hold {longest} tokens, the cache has room for {self.capacity}")
        want = [s * n_tok + n_tok - 1 for s in range(n_seq)] if want is None else list(want)
        if any(not 0 <= r < n_seq * n_tok for r in want):
            raise ValueError("a wanted row is outside the step")
        if self.graphs and n_tok == 1 and not trace and want == list(range(n_seq)):
            logits = self._decode(slots, ids, longest)
        else:
            logits = self._eager(slots, ids, want, longest, trace)
        for s in slots:
            self.length[s] += n_tok
        return logits

    def _eager(self, slots, ids, want, longest, trace):
        n_seq, n_tok = ids.shape
        # the wanted rows are read in blocks no longer than the step itself, so repeated rows do not matter
        dev = torch.tensor(list(slots) + want, dtype=torch.int32).cuda(non_blocking=True)
        tokens = ids.cuda(non_blocking=True)
        need = self._workspace_bytes(n_seq, n_tok, longest)
        if self.workspace.numel() < need:
            self.workspace = torch.empty(need, dtype=torch.uint8, device="cuda")
        hidden = torch.empty((self.n_layers, n_seq * n_tok, self.width), device="cuda") if trace else None
        logits = torch.empty((len(want), self.vocab), device="cuda")
        if len(want) > n_seq * n_tok:
            raise ValueError("more wanted rows than rows")
        self._enqueue(dev, n_seq, n_tok, longest, tokens, dev[n_seq:], len(want), logits, hidden, self.workspace)
        return (logits, hidden) if trace else logits

    def _decode(self, slots, ids, longest):
        """One token per sequence, replayed from a graph per (sequences, context class): the context bounds the split
        of the attention over the cache, so it is rounded up to a power of two."""
        n_seq = len(slots)
        context = min(self.capacity, max(64, 1 << (longest - 1).bit_length()))
        key = (n_seq, context)
        if key not in self._graphs:
            if len(self._graphs) >= self.MAX_GRAPHS:
                self._graphs.pop(next(iter(self._graphs)))
            self._graphs[key] = self._capture(n_seq, context)
        graph, inputs, logits, _, _ = self._graphs[key]
        inputs.copy_(torch.cat([torch.tensor(list(slots), dtype=torch.int32), ids.reshape(-1)]), non_blocking=True)
        graph.replay()
        return logits.clone()

    def _capture(self, n_seq: int, context: int):
        inputs = torch.zeros(2 * n_seq, dtype=torch.int32, device="cuda")
        rows = torch.arange(n_seq, dtype=torch.int32, device="cuda")
        logits = torch.empty((n_seq, self.vocab), device="cuda")
        workspace = torch.empty(self._workspace_bytes(n_seq, 1, context), dtype=torch.uint8, device="cuda")
        torch.cuda.synchronize()
        before = self.L.tbl_launch_count()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            self._enqueue(inputs, n_seq, 1, context, inputs[n_seq:], rows, n_seq, logits, None, workspace)
        self.launches_per_step = int(self.L.tbl_launch_count() - before)
        return graph, inputs, logits, rows, workspace

    def feed(self, slot: int, tokens: Sequence[int], want: Optional[Sequence[int]] = None) -> torch.Tensor:
        """Any number of tokens of one sequence, in portions; logits of the wanted places (default: the last)."""
        want = [len(tokens) - 1] if want is None else list(want)
        parts, order = [], []
        for lo in range(0, len(tokens), self.PORTION):
            part = list(tokens[lo:lo + self.PORTION])
            at = [k for k, r in enumerate(want) if lo <= r < lo + len(part)]
            places = sorted({want[k] - lo for k in at})
            logits = self.step([slot], [part], places)
            row = {r: n for n, r in enumerate(places)}
            parts.append(logits[[row[want[k] - lo] for k in at]] if at else logits[:0])
            order += at
        out = torch.cat(parts)
        return out if order == sorted(order) else out[torch.tensor(order).argsort()]

    def device_status(self) -> int:
        """The library's sticky status word (synchronises): 0, or an OR of TBL_DEV_* codes."""
        return self.L.tbl_device_status(self._stream())


def load(folder: str, dtype: str = "bfloat16", slots: int = 1, capacity: int = 1024, cfg: Optional[dict] = None) -> StackEngine:
    """Engine over a checkpoint folder."""
    return StackEngine(cfg or read_config(folder), read_safetensors(os.path.join(folder, "model.safetensors")), dtype, slots,
                       capacity)
