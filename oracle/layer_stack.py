"""Plain numpy (float64) restatement of the layer-stack designs: one function per mechanism, one token or one
query at a time, no blocking, no cache tricks.  Test infrastructure only: nothing in `reimagined_b200/` imports
this file, and it imports nothing from there.

A model is a configuration dict plus a dict of named weight arrays; `Decoder` runs it token by token or in
portions, with the recurrent states and the latent caches of one sequence.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import numpy as np

F = np.float64


def sigmoid(z):
    z = np.asarray(z, F)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    z = np.asarray(z, F)
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def linear(x, w, b=None):
    """Rows of x times W^T; W is stored [out, in]."""
    y = np.asarray(x, F) @ np.asarray(w, F).T
    return y if b is None else y + np.asarray(b, F)


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis, times w (None: no weight)."""
    x = np.asarray(x, F)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * np.asarray(w, F)


def dynamic_tanh(x, alpha, w, b):
    """tanh(alpha x) w + b: a norm without statistics."""
    return np.tanh(F(alpha) * np.asarray(x, F)) * np.asarray(w, F) + np.asarray(b, F)


def embed(table, tokens, scale):
    return np.asarray(table, F)[np.asarray(tokens)] * scale


def rotate_half(x, positions, base, dims):
    """Rotary positions on the first `dims` entries of the last axis; entry i goes with entry i + dims/2.
    x [T, ..., n], positions [T]."""
    x = np.array(x, F)
    half = dims // 2
    freq = F(base) ** (-2.0 * np.arange(half) / dims)
    ang = np.asarray(positions, F)[:, None] * freq[None, :]
    ang = ang.reshape((len(positions),) + (1,) * (x.ndim - 2) + (half,))
    u, v = x[..., :half].copy(), x[..., half:dims].copy()
    x[..., :half] = u * np.cos(ang) - v * np.sin(ang)
    x[..., half:dims] = v * np.cos(ang) + u * np.sin(ang)
    return x


def unit(k):
    return k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + 1e-6)


def delta_decay(h, w1, w2, w0):
    """Decay per channel, in (exp(-exp(-1/2)), 1)."""
    z = linear(np.tanh(linear(h, w1)), w2) + np.asarray(w0, F)
    return np.exp(-np.exp(-0.5) * sigmoid(z))


def delta_step(S, r, k, v, w, a):
    """One token of the generalized delta rule of one head: state [key, value] -> (new state, output)."""
    u = unit(k)
    S = w[:, None] * S - np.outer(a * u, u @ S) + np.outer(k, v)
    return S, S.T @ r


def general_delta(h, P, p, cfg, eps, states):
    """Mixer: h [T, width]; states [heads, dim, dim] is updated in place."""
    H, d = cfg["heads"], cfg["dim"]
    T = len(h)
    r, k, v = (linear(h, P[p + n]).reshape(T, H, d) for n in ("r", "k", "v"))
    w = delta_decay(h, P[p + "w1"], P[p + "w2"], P[p + "w0"]).reshape(T, H, d)
    a = sigmoid(linear(h, P[p + "a"], P[p + "a.b"])).reshape(T, H, d)
    o = np.zeros((T, H, d))
    for t in range(T):
        for n in range(H):
            states[n], o[t, n] = delta_step(states[n], r[t, n], k[t, n], v[t, n], w[t, n], a[t, n])
    o = rms_norm(o, None, eps).reshape(T, H * d) * np.asarray(P[p + "norm"], F)
    return linear(o * sigmoid(linear(h, P[p + "g"])), P[p + "o"])


def softmax_attention(q, keys, values, scale):
    """One query over all given keys: q [n], keys [m, n], values [m, vdim]."""
    s = keys @ q * scale
    e = np.exp(s - s.max())
    return (e / e.sum()) @ values


def latent_attention(h, P, p, cfg, eps, cache):
    """Mixer: h [T, width]; cache is a list of (latent, rotated key part), one entry per earlier token."""
    H, d, rd, vd, R = (cfg[n] for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    T, first = len(h), len(cache)
    pos = np.arange(first, first + T)
    base, dims = cfg["rot"]["base"], cfg["rot"]["dims"]
    q = linear(rms_norm(linear(h, P[p + "dq"]), P[p + "dq.norm"], eps), P[p + "uq"]).reshape(T, H, d + rd)
    q_plain, q_rot = q[..., :d], rotate_half(q[..., d:], pos, base, dims)
    kv = linear(h, P[p + "dkv"])
    c = rms_norm(kv[:, :R], P[p + "dkv.norm"], eps)
    k_rot = rotate_half(kv[:, R:], pos, base, dims)
    cache.extend(zip(c, k_rot))
    lat = np.array([e[0] for e in cache])
    rot = np.array([e[1] for e in cache])
    keys = linear(lat, P[p + "uk"]).reshape(-1, H, d)
    values = linear(lat, P[p + "uv"]).reshape(-1, H, vd)
    out = np.zeros((T, H, vd))
    for t in range(T):
        n = first + t + 1
        for i in range(H):
            k_full = np.concatenate([keys[:n, i], rot[:n]], axis=1)
            out[t, i] = softmax_attention(np.concatenate([q_plain[t, i], q_rot[t, i]]), k_full, values[:n, i], cfg["scale"])
    return linear(out.reshape(T, H * vd) * sigmoid(linear(h, P[p + "g"])), P[p + "o"])


def query_temperature(position, coef, every):
    return 1.0 + coef * np.log(np.floor((position + 1) / every) + 1.0)


def differential_lambda(P, p, diff):
    dot = lambda a, b: float(np.sum(np.asarray(P[p + a], F) * np.asarray(P[p + b], F)))
    return np.exp(dot("lq1", "lk1")) - np.exp(dot("lq2", "lk2")) + diff


def differential_output(a1, a2, lam, diff, eps):
    return rms_norm(a1 - lam * a2, None, eps) * (1.0 - diff)


def grouped_attention(h, P, p, cfg, eps, cache):
    """Mixer: h [T, width]; cache is a list of (keys [G, maps, dim], values [G, vdim]), one entry per token of the sequence
    so far.  A layer without a key projection finds the step's own tokens in it already.  With "diff" in the configuration
    every head has two maps, whose difference is normed (differential attention)."""
    H, G, d, vd = (cfg[n] for n in ("heads", "kv_heads", "dim", "vdim"))
    T, maps = len(h), 2 if "diff" in cfg else 1
    project = lambda name: linear(h, P[p + name], P.get(p + name + ".b"))
    q = project("q").reshape(T, H, maps, d)
    if p + "k" in P:
        cache.extend(zip(project("k").reshape(T, G, maps, d), project("v").reshape(T, G, vd)))
    first = len(cache) - T
    keys, values = np.array([e[0] for e in cache]), np.array([e[1] for e in cache])
    o = np.zeros((T, H, vd))
    for t in range(T):
        n, temp = first + t + 1, 1.0
        if "q_temp" in cfg:
            temp = query_temperature(first + t, cfg["q_temp"]["coef"], cfg["q_temp"]["every"])
        for i in range(H):
            g = i // (H // G)
            a = [softmax_attention(q[t, i, m] * temp, keys[:n, g, m], values[:n, g], cfg["scale"]) for m in range(maps)]
            o[t, i] = a[0] if maps == 1 else differential_output(a[0], a[1], differential_lambda(P, p, cfg["diff"]), cfg["diff"], eps)
    o = o.reshape(T, H * vd)
    if p + "g" in P:
        o = o * sigmoid(linear(h, P[p + "g"]))
    return linear(o, P[p + "o"], P.get(p + "o.b"))


def streams_in(streams, weights):
    """A sublayer's input: the weighted sum of the residual streams."""
    return sum(F(w) * x for w, x in zip(np.asarray(weights, F), streams))


def streams_out(streams, mix, out, y):
    """The residual streams after a sublayer whose result is y; mix is indexed [from, to]."""
    mix, out = np.asarray(mix, F), np.asarray(out, F)
    return [sum(mix[s, t] * streams[s] for s in range(len(streams))) + out[t] * y for t in range(len(streams))]


def gelu_ff(h, P, p):
    return linear(gelu_tanh(linear(h, P[p + "gate"])) * linear(h, P[p + "up"]), P[p + "down"])


def dense_ff(h, P, p):
    g = linear(h, P[p + "gate"], P[p + "gate.b"])
    u = linear(h, P[p + "up"], P[p + "up.b"])
    return linear(silu(g) * u, P[p + "down"], P[p + "down.b"])


def depth_average(weights, xs):
    return sum(F(w) * x for w, x in zip(np.asarray(weights, F), xs))


class Decoder:
    """One sequence through the stack; `feed` takes any number of tokens and returns their logits."""

    def __init__(self, cfg: dict, params: Dict[str, np.ndarray]):
        self.cfg, self.P = cfg, params
        self.memory: List = []
        for layer in cfg["layers"]:
            m = layer["mixer"]
            self.memory.append(np.zeros((m["heads"], m["dim"], m["dim"])) if layer["type"] == "general_delta" else [])

    def feed(self, tokens, trace: Optional[list] = None):
        cfg, P, eps = self.cfg, self.P, self.cfg["norm"]["eps"]
        x = embed(P["embed"], tokens, cfg["embedding"]["scale"])
        xs = [x]
        mixers = {"general_delta": general_delta, "latent_attention": latent_attention}
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            x = x + mixers[layer["type"]](rms_norm(x, P[p + "norm1"], eps), P, p + "mix.", layer["mixer"], eps, self.memory[i])
            if layer["mlp"] is not None:
                x = x + dense_ff(rms_norm(x, P[p + "norm2"], eps), P, p + "mlp.")
            xs.append(x)
            x = depth_average(P[p + "dwa"], xs)
            if trace is not None:
                trace.append(x.copy())
        return linear(rms_norm(x, P["final.norm"], eps), P["embed"])


class StreamDecoder:
    """The same for the design with several residual streams, Dynamic Tanh norms and differential attention (Goguvik)."""

    def __init__(self, cfg: dict, params: Dict[str, np.ndarray]):
        self.cfg, self.P = cfg, params
        self.memory: List[list] = []
        for layer in cfg["layers"]:
            source = layer["mixer"].get("kv_from")
            self.memory.append([] if source is None else self.memory[source])

    def feed(self, tokens, trace: Optional[list] = None):
        cfg, P, eps = self.cfg, self.P, self.cfg["norm"]["eps"]
        norm = lambda x, name: dynamic_tanh(x, P[name + ".alpha"], P[name], P[name + ".b"])
        xs = [embed(P["embed"], tokens, 1.0)] * cfg["streams"]
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            sublayers = [lambda h: grouped_attention(h, P, p + "mix.", layer["mixer"], eps, self.memory[i])]
            if layer["mlp"] is not None:
                sublayers.append(lambda h: gelu_ff(h, P, p + "mlp."))
            for n, sublayer in enumerate(sublayers, 1):
                hc = f"{p}hc{n}."
                y = sublayer(norm(streams_in(xs, P[hc + "in"]), f"{p}norm{n}"))
                xs = streams_out(xs, P[hc + "mix"], P[hc + "out"], y)
            if trace is not None:
                trace.append(sum(xs))
        return linear(norm(sum(xs), "final.norm"), P["embed"])


def decoder(cfg: dict, params: Dict[str, np.ndarray]):
    return (StreamDecoder if "streams" in cfg else Decoder)(cfg, params)
