"""Layer-stack models, the parts that need no GPU: the oracle against itself, checkpoints, configuration checks, sampling,
the generation loop, and what the C entry points refuse."""
import json
import os
import re

import numpy as np
import pytest
import torch

import stack_helpers as S
from oracle import layer_stack as O

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", ["odd", "only_delta", "only_latent", "diff_odd", "diff_wide"])
def test_oracle_does_not_depend_on_the_cut(name):
    _, p = S.weights(name)
    ids = S.tokens(name, 23)
    whole = O.decoder(S.CONFIGS[name], p).feed(ids)
    d = O.decoder(S.CONFIGS[name], p)
    parts, at = [], 0
    for n in (1, 2, 7, 1, 12):
        parts.append(d.feed(ids[at:at + n]))
        at += n
    np.testing.assert_allclose(np.concatenate(parts), whole, rtol=1e-9, atol=1e-9)


def test_oracle_delta_step_by_hand():
    # two keys, one value: S = diag(w) S - (a*u)(u.S) + k v
    s, o = O.delta_step(np.array([[2.0], [1.0]]), np.array([1.0, -1.0]), np.array([3.0, 4.0]), np.array([0.5]),
                        np.array([0.9, 0.8]), np.array([0.25, 0.5]))
    u = np.array([3.0, 4.0]) / np.sqrt(25.0 + 1e-6)
    us = u[0] * 2 + u[1] * 1
    want = np.array([0.9 * 2 - 0.25 * u[0] * us + 1.5, 0.8 * 1 - 0.5 * u[1] * us + 2.0])
    np.testing.assert_allclose(s[:, 0], want)
    np.testing.assert_allclose(o, [want[0] - want[1]])


def test_oracle_rotation_pairs_and_angle():
    x = np.arange(1.0, 9.0)[None]
    y = O.rotate_half(x, [3], 10.0, 6)
    a = 3 * 10.0 ** (-2 / 6)
    np.testing.assert_allclose(y[0, 1], 2 * np.cos(a) - 5 * np.sin(a))
    np.testing.assert_allclose(y[0, 4], 5 * np.cos(a) + 2 * np.sin(a))
    np.testing.assert_allclose(y[0, 6:], x[0, 6:])


def test_oracle_streams_and_norm_by_hand():
    xs, y = [np.array([[1.0, 2.0]]), np.array([[-3.0, 0.5]])], np.array([[10.0, 20.0]])
    np.testing.assert_allclose(O.streams_in(xs, [2.0, 3.0]), [[-7.0, 5.5]])
    got = O.streams_out(xs, [[1.0, 0.5], [0.25, 2.0]], [0.1, 0.2], y)              # mix[from][to]
    np.testing.assert_allclose(got[0], [[1.0 - 0.75 + 1.0, 2.0 + 0.125 + 2.0]])
    np.testing.assert_allclose(got[1], [[0.5 - 6.0 + 2.0, 1.0 + 1.0 + 4.0]])
    np.testing.assert_allclose(O.dynamic_tanh([2.0], 0.25, [3.0], [1.0]), [3 * np.tanh(0.5) + 1])
    np.testing.assert_allclose(O.gelu_tanh([1.0, -2.0]), [0.841192, -0.045402], atol=1e-6)


def test_oracle_query_temperature_steps():
    assert [round(float(O.query_temperature(p, 2.0, 4)), 6) for p in (0, 2, 3, 6, 7)] == [
        1.0, 1.0, round(1 + 2 * np.log(2), 6), round(1 + 2 * np.log(2), 6), round(1 + 2 * np.log(3), 6)]


def test_oracle_differential_attention_by_hand():
    """One head, one-dimensional keys, two tokens."""
    cfg = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 2, "scale": 0.5, "diff": 0.25, "q_temp": {"coef": 1.0, "every": 2}}
    P = {"q": [[1.0], [2.0]], "q.b": [0.0, 0.5], "k": [[1.0], [-1.0]], "k.b": [0.25, 0.0], "v": [[1.0], [0.0]], "v.b": [0.0, 3.0],
         "lq1": [0.5], "lk1": [1.0], "lq2": [0.0], "lk2": [1.0], "g": np.zeros((2, 1)), "o": np.eye(2), "o.b": [0.0, 1.0]}
    h = np.array([[1.0], [2.0]])
    t = 1 + np.log(2)                                                               # the second token: (1 + 1) / 2 = 1
    s1, s2 = 0.5 * t * 2.0 * np.array([1.25, 2.25]), 0.5 * t * 4.5 * np.array([-1.0, -2.0])
    a1, a2 = (np.exp(s) / np.exp(s).sum() @ np.array([[1.0, 3.0], [2.0, 3.0]]) for s in (s1, s2))
    o = a1 - (np.exp(0.5) - 1 + 0.25) * a2
    o = o / np.sqrt((o ** 2).mean() + 1e-3) * 0.75
    np.testing.assert_allclose(O.grouped_attention(h, P, "", cfg, 1e-3, [])[1], 0.5 * o + [0.0, 1.0])


def test_safetensors_round_trip_at_any_offset(tmp_path):
    from reimagined_b200.checkpoint import read_safetensors, write_safetensors
    want = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32), "c": torch.tensor(2.5), "e": torch.zeros(0, 4)}
    path = str(tmp_path / "t.safetensors")
    write_safetensors(path, want)
    got = read_safetensors(path)
    assert set(got) == set(want) and all(torch.equal(got[k], want[k]) and got[k].dtype == want[k].dtype for k in want)
    raw = open(path, "rb").read()
    n = int.from_bytes(raw[:8], "little")
    head = raw[8:8 + n].rstrip() + b" "                      # the data starts at an odd place now
    if len(head) % 2 == 0:
        head += b" "
    open(path, "wb").write(len(head).to_bytes(8, "little") + head + raw[8 + n:])
    got = read_safetensors(path)
    assert all(torch.equal(got[k], want[k]) for k in want)
    open(path, "wb").write(raw[:-3])
    with pytest.raises(ValueError):
        read_safetensors(path)


def test_weights_must_fit_the_configuration():
    from reimagined_b200.stack import check_weights
    w, _ = S.weights("odd")
    check_weights(S.ODD, w)
    for change in (lambda d: d.pop("l1.mix.w0"), lambda d: d.update(extra=torch.zeros(1)),
                   lambda d: d.update({"l0.mix.uk": d["l0.mix.uk"][:-1]})):
        d = dict(w)
        change(d)
        with pytest.raises(ValueError):
            check_weights(S.ODD, d)
    for path, value in ((("layers", 0, "type"), "no_such_mixer"), (("layers", 0, "mlp"), {"kind": "sparse", "ff": 8})):
        cfg = json.loads(json.dumps(S.ODD))
        node = cfg
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ValueError):
            check_weights(cfg, w)


def test_weights_of_layers_that_share_a_cache():
    from reimagined_b200.stack import check_weights
    w, _ = S.weights("diff_odd")
    assert "l0.mix.k.b" in w and "l1.mix.k" not in w and "l1.mix.v.b" not in w and "l1.hc2.mix" not in w and "l3.hc1.mix" in w
    check_weights(S.DIFF_ODD, w)
    # tensors around a feed-forward that is not there may be in the file
    check_weights(S.DIFF_ODD, {**w, "l1.norm2": w["l0.norm2"], "l1.hc2.in": w["l0.hc2.in"]})
    for name, value in (("l1.mix.k", w["l0.mix.k"]), ("l0.dwa", torch.ones(2)), ("l0.mlp.gate.b", torch.zeros(50)), ("l0.hc1.mix", torch.zeros(3, 2)),
                        ("l2.norm1.alpha", torch.zeros(1)), ("final.norm.b", None)):
        d = {**w, name: value}
        if value is None:
            del d[name]
        with pytest.raises(ValueError):
            check_weights(S.DIFF_ODD, d)


def test_query_temperature_table():
    from reimagined_b200.stack import StackEngine

    class Stub:
        capacity, _temperatures, f32 = 300, {}, staticmethod(lambda t: t.numpy())
    for coef, every in ((0.7, 7), (1.5, 1), (0.3, 64), (0.4, 2.5)):
        np.testing.assert_allclose(StackEngine.query_temperature(Stub, coef, every), O.query_temperature(np.arange(300), coef, every))


def test_registry_knows_its_models(tmp_path):
    from reimagined_b200 import registry
    (tmp_path / "config.json").write_text(json.dumps(S.ODD))
    e, cfg = registry.entry(str(tmp_path))
    assert e.library == "stack" and "float32" in e.dtypes and cfg == S.ODD
    (tmp_path / "config.json").write_text(json.dumps(S.DIFF_ODD))
    assert registry.entry(str(tmp_path))[0].dtypes == ("bfloat16", "float32")
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nonesuch"}))
    with pytest.raises(ValueError):
        registry.entry(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "JambaHybrid"}))
    with pytest.raises(ValueError):
        registry.load(str(tmp_path), "float32")


def test_sampling():
    from reimagined_b200.generate import sample
    z = torch.tensor([[0.0, 3.0, 1.0, 2.9], [5.0, -1.0, 5.0, 0.0]])
    assert sample(z).tolist() == [1, 0]
    gen = torch.Generator().manual_seed(0)
    draws = torch.stack([sample(z, 1.0, generator=gen) for _ in range(300)])
    assert set(draws[:, 0].tolist()) >= {1, 3}
    assert set(torch.stack([sample(z, 1.0, top_k=2, generator=gen) for _ in range(100)])[:, 0].tolist()) == {1, 3}
    assert set(torch.stack([sample(z, 1.0, top_p=0.4, generator=gen) for _ in range(50)])[:, 0].tolist()) == {1}
    assert set(torch.stack([sample(z, 1.0, top_p=0.9, generator=gen) for _ in range(100)])[:, 0].tolist()) == {1, 3}


class CountingEngine:
    """Next token = (sum of the sequence's tokens) mod vocab; checks how slots are used."""

    vocab, capacity = 11, 40

    def __init__(self, slots):
        self.slots, self.seq, self.batches = slots, {}, []

    def open(self):
        slot = next(i for i in range(self.slots) if i not in self.seq)
        self.seq[slot] = []
        return slot

    def close(self, slot):
        del self.seq[slot]

    def _logits(self, slot):
        return torch.nn.functional.one_hot(torch.tensor([sum(self.seq[slot]) % self.vocab]), self.vocab).float()

    def feed(self, slot, tokens, want=None):
        self.seq[slot] += tokens
        return self._logits(slot)

    def step(self, slots, tokens):
        self.batches.append(len(slots))
        return torch.cat([self.feed(s, t) for s, t in zip(slots, tokens)])


def test_generation_admits_batches_and_retires():
    from reimagined_b200.generate import generate

    def alone(prompt, n, stop=()):
        seq, new = list(prompt), []
        while len(new) < n and not (new and new[-1] in stop):
            new.append(sum(seq) % 11)
            seq.append(new[-1])
        return new

    prompts = [[1, 2], [5], [3, 3, 3], [10], [7, 1]]
    e = CountingEngine(2)
    assert generate(e, prompts, 6) == [alone(p, 6) for p in prompts] and not e.seq and max(e.batches) == 2
    e = CountingEngine(3)
    assert generate(e, prompts, 9, stop=[4, 9]) == [alone(p, 9, (4, 9)) for p in prompts] and not e.seq
    assert generate(CountingEngine(1), [[1]], 0) == [[]]
    with pytest.raises(ValueError):
        generate(CountingEngine(1), [[1] * 30], 20)


def test_library_exports_every_declared_symbol(stack_lib):
    from reimagined_b200 import capi
    with open(os.path.join(ROOT, "include", "layer_stack.h")) as f:
        names = set(re.findall(r"\b(tbl_[a-z0-9_]+)\s*\(", f.read()))
    assert names == set(capi.STACK_SYMBOLS)
    assert all(hasattr(stack_lib, n) for n in names)


def test_entry_points_refuse_before_they_touch_a_device(stack_lib):
    import ctypes as C
    from reimagined_b200 import capi
    L = stack_lib
    d = capi.DeltaMixer()
    d.in_ = capi.DenseView(4096, 4096, 64, 5 * 32 + 8)
    d.decay_up, d.out = capi.DenseView(4096, 4096, 8, 32), capi.DenseView(4096, None, 32, 64)
    d.norm, d.heads, d.dim, d.rank = 4096, 2, 16, 8
    layer = capi.StackLayer()
    layer.mixer, layer.norm1, layer.delta = capi.MIXER_GENERAL_DELTA, 4096, d
    m = capi.StackModel(64, 100, 1, 4096, 1.0, 1e-5, C.pointer(layer), 4096, capi.DenseView(4096, None, 64, 100))
    size = L.tbl_stack_state_bytes(C.byref(m), capi.BF16, 2, 16)
    assert size >= 2 * 2 * 16 * 16 * 4
    step = lambda **k: L.tbl_stack_step(C.byref(m), k.get("precision", 1), 2, 16, k.get("state", 4096), 4096, k.get("n_seq", 1),
                                        k.get("n_tok", 1), k.get("context", 16), 4096, 4096, k.get("n_want", 1), 4096, None,
                                        k.get("ws", 4096), k.get("ws_bytes", 1 << 40), None)
    assert step(precision=7) == -1 and step(n_seq=3) == -1 and step(context=17) == -1 and step(n_tok=9, context=8) == -1
    assert step(n_want=2) == -1 and step(state=None) == -1
    assert step(ws_bytes=16) == -7 and step(ws=4096 + 16) == -6
    d.dim = 300
    layer.delta = d
    assert step() == -2 and L.tbl_stack_state_bytes(C.byref(m), capi.BF16, 2, 16) == 0
    layer.mixer = 9
    assert step() == -10
    v = capi.DenseView(4096, None, 64, 32)
    assert L.tbl_dense_forward(C.byref(v), 1, 0, None, 64, 1, None, 4096, None) == -1
    assert L.tbl_dense_forward(C.byref(v), 1, 0, 4096, 63, 1, None, 4096, None) == -1
    assert L.tbl_gated_dense_forward(C.byref(v), 1, 0, 4096, 64, 1, 8, 4096, None) == -2
    v.weight = 4100
    assert L.tbl_dense_forward(C.byref(v), 1, 0, 4096, 64, 1, None, 4096, None) == -6


def test_models_with_streams_are_checked(stack_lib):
    import ctypes as C
    from reimagined_b200 import capi
    L = stack_lib

    def layer(kv_from=-1, heads=4, kv_heads=2, dim=16, vdim=24):
        a, l = capi.AttentionMixer(), capi.StackLayer()
        kv = kv_heads * (2 * dim + vdim) if kv_from < 0 else 0
        a.in_, a.out = capi.DenseView(4096, 4096, 64, heads * (2 * dim + vdim) + kv), capi.DenseView(4096, 4096, heads * vdim, 64)
        a.heads, a.kv_heads, a.dim, a.vdim, a.maps, a.gated, a.kv_from, a.scale, a.out_scale = heads, kv_heads, dim, vdim, 2, 1, kv_from, 0.1, 0.5
        l.mixer, l.norm1, l.attention, l.tanh1, l.hyper1 = capi.MIXER_ATTENTION, 4096, a, capi.TanhNorm(4096, 0.5), capi.Hyper(4096, 4096, 4096)
        return l

    def state_bytes(layers, precision=capi.BF16, norm=capi.NORM_DYNAMIC_TANH, streams=2):
        arr = (capi.StackLayer * len(layers))(*layers)
        m = capi.StackModel(64, 100, len(layers), 4096, 1.0, 1e-5, arr, 4096, capi.DenseView(4096, None, 64, 100), norm, capi.TanhNorm(4096, 0.5), streams)
        return L.tbl_stack_state_bytes(C.byref(m), precision, 3, 50)

    one = state_bytes([layer()])
    # a token's row: two keys of 16 and values of 24, padded to 32, for every key/value head
    assert one == 256 + -(-3 * 50 * 2 * 64 * 2 // 256) * 256
    assert state_bytes([layer(), layer(0)]) == one                        # no cache of its own
    assert state_bytes([layer(), layer(0), layer()]) == 2 * one - 256
    assert state_bytes([layer()], capi.F32) == 2 * one - 256
    assert state_bytes([layer()], streams=8) and not state_bytes([layer()], streams=9) and not state_bytes([layer()], norm=5)
    assert not state_bytes([layer(0)])                                    # itself
    assert not state_bytes([layer(1), layer()])                           # a later layer
    assert not state_bytes([layer(), layer(0), layer(1)])                 # a layer that shares
    assert not state_bytes([layer(), layer(0, kv_heads=4)]) and not state_bytes([layer(), layer(0, vdim=16)])
    assert not state_bytes([layer(heads=5)]) and not state_bytes([layer(dim=600)])
    bare = layer()
    bare.hyper1.mix = None
    assert not state_bytes([bare])
    averaged = layer()
    averaged.depth_weights = 4096
    assert not state_bytes([averaged])


def test_attention_entry_points_refuse_before_they_touch_a_device(stack_lib):
    import ctypes as C
    from reimagined_b200 import capi
    L, a = stack_lib, capi.AttentionMixer()
    a.in_, a.out = capi.DenseView(4096, None, 8, 4 * 32 + 2 * 56), capi.DenseView(4096, None, 4 * 24, 8)
    a.heads, a.kv_heads, a.dim, a.vdim, a.maps, a.kv_from, a.scale, a.out_scale = 4, 2, 16, 24, 2, -1, 0.1, 1.0
    assert L.tbl_attention_cache_width(C.byref(a)) == 64
    run = lambda **k: L.tbl_attention_forward(C.byref(a), k.get("precision", 1), k.get("route", 0), 1e-5, 4096, k.get("cache", 4096), k.get("slots", 2), 16, 4096,
                                              4096, k.get("n_seq", 1), k.get("n_tok", 1), k.get("context", 16), 4096, k.get("ws", 4096), k.get("bytes", 1 << 40), None)
    assert run(precision=3) == -1 and run(context=17) == -1 and run(n_tok=9, context=8) == -1 and run(cache=None) == -1 and run(n_seq=3) == -1
    assert run(bytes=0) == -7 and run(ws=4096 + 16) == -6 and run(cache=4096 + 8) == -6
    a.kv_heads = 3
    assert run() == -2 and L.tbl_attention_cache_width(C.byref(a)) == 0
    norm = lambda **k: L.tbl_stream_norm(4096, k.get("stride", 64), k.get("streams", 2), k.get("y", 4096), 4096, k.get("out", 4096), k.get("store", 0), 4096, 1,
                                         k.get("index"), 1, 64, k.get("kind", 1), 1e-5, 0.5, 4096, k.get("bias", 4096), None, 4096, None)
    assert norm(streams=0) == -1 and norm(streams=9) == -10 and norm(out=None) == -1 and norm(kind=2) == -1 and norm(bias=None) == -1
    assert norm(index=4096, store=1) == -1 and norm(stride=66) == -6 and norm(y=4100) == -6
