"""Layer-stack models through the engine, the scheduler and the command line, against the plain oracle and against
themselves under other schedules."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import stack_helpers as S

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module", autouse=True)
def _built(cuda, stack_lib):
    return stack_lib


_cache = {}


def setup(name, dtype, n=150):
    """(engine, token ids, oracle logits), made once."""
    if (name, dtype) not in _cache:
        _cache[name, dtype] = S.engine(name, dtype)
    if name not in _cache:
        ids = S.tokens(name, n)
        _cache[name] = ids, S.oracle_logits(name, _cache[name, dtype][1], ids)
    return (_cache[name, dtype][0],) + _cache[name]


def run(e, ids, cuts):
    """Logits of every place, the tokens fed in the given portions."""
    import torch
    slot, at, out = e.open(), 0, []
    for n in cuts:
        out.append(e.feed(slot, ids[at:at + n], list(range(n))).clone())
        at += n
    assert at == len(ids) and e.device_status() == 0
    e.close(slot)
    return torch.cat(out)


DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(S.CONFIGS))
def test_prompt_matches_oracle(name, dtype):
    e, ids, want = setup(name, dtype)
    S.close(run(e, ids, [len(ids)]), want, dtype)


@pytest.mark.parametrize("name", ["odd", "even", "diff_odd", "diff_even"])
def test_residual_stream_after_every_layer(name):
    from oracle.layer_stack import decoder
    e, p = S.engine(name)
    ids, layers = S.tokens(name, 30, 4), []
    decoder(S.CONFIGS[name], p).feed(ids, layers)
    slot = e.open()
    _, hidden = e.step([slot], [ids], trace=True)
    for got, want in zip(hidden.cpu().numpy(), layers):
        assert np.abs(got - want).max() <= 2e-5 * np.abs(want).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(S.CONFIGS))
def test_token_by_token_matches_oracle(name, dtype):
    e, ids, want = setup(name, dtype)
    S.close(run(e, ids[:70], [1] * 70), want[:70], dtype)
    S.close(run(e, ids, [110] + [1] * 40), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even", "wide", "diff_odd", "diff_even", "diff_wide"])
@pytest.mark.parametrize("cuts", [[2] * 75, [37, 2, 3, 1, 64, 2, 41], [3, 48, 47, 49, 3], [16, 1, 15, 17, 1, 100], [128, 2, 20], [149, 1]])
def test_portions_match_oracle(name, dtype, cuts):
    e, ids, want = setup(name, dtype)
    S.close(run(e, ids, cuts), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["even", "diff_even"])
def test_long_prompt_in_engine_portions_and_the_order_of_wanted_places(name, dtype):
    e, ids, want = setup(name, dtype)
    e.PORTION = 48
    try:
        slot, places = e.open(), [149, 3, 47, 48, 3, 96, 0]
        got = e.feed(slot, ids, places)
        e.close(slot)
    finally:
        del e.PORTION
    S.close(got, want[places], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even", "diff_odd", "diff_even"])
def test_unequal_sequences_decoded_together_match_each_alone(name, dtype):
    import torch
    e, p = S.engine(name, dtype)
    prompts = [S.tokens(name, n, n) for n in (5, 90, 33)]
    more = np.random.default_rng(9).integers(0, S.CONFIGS[name]["vocab"], (12, 3))
    slots = [e.open() for _ in prompts]
    for s, ids in zip(slots, prompts):
        e.feed(s, ids)
    got = torch.stack([e.step(slots, [[int(t)] for t in row]) for row in more[:6]])
    # another order of the same slots, and fewer of them
    got2 = torch.stack([e.step(slots[::-1], [[int(t)] for t in row[::-1]]).flip(0) for row in more[6:9]])
    got3 = torch.stack([e.step([slots[1]], [[int(row[1])]])[0] for row in more[9:]])
    for i, ids in enumerate(prompts):
        want = S.oracle_logits(name, p, ids + more[:, i].tolist())[len(ids):]
        S.close(torch.cat([got[:, i], got2[:, i]]), want[:9], dtype)
        if i == 1:
            S.close(got3, want[9:], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["even", "diff_even"])
def test_prompts_in_lockstep_match_each_alone(name, dtype):
    e, p = S.engine(name, dtype)
    a, b = S.tokens(name, 120, 1), S.tokens(name, 120, 2)
    slots = [e.open(), e.open()]
    e.feed(slots[1], b[:20])
    got = e.step(slots, [a[:60], b[20:80]], list(range(120)))
    S.close(got[:60], S.oracle_logits(name, p, a[:60]), dtype)
    S.close(got[60:], S.oracle_logits(name, p, b[:80])[20:], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even", "diff_odd", "diff_even"])
def test_slots_used_again_start_empty(name, dtype):
    e, ids, want = setup(name, dtype)
    run(e, S.tokens(name, 390, 77), [390])
    for cuts in ([150], [1] * 3 + [147], [2, 148]):
        S.close(run(e, ids, cuts), want, dtype)
    # while a neighbour holds a long sequence
    other = e.open()
    e.feed(other, S.tokens(name, 300, 5))
    S.close(run(e, ids, [149, 1]), want, dtype)
    e.close(other)


@pytest.mark.parametrize("name", ["even", "diff_even"])
def test_the_same_bits_whatever_else_is_live(name):
    e, ids, _ = setup(name, "bfloat16")
    first = run(e, ids, [100] + [1] * 50)
    other = e.open()
    e.feed(other, S.tokens(name, 217, 5))
    assert (run(e, ids, [100] + [1] * 50) == first).all()
    e.close(other)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["even", "diff_even"])
def test_long_decode(name, dtype):
    e, p = S.engine(name, dtype, slots=1, capacity=700)
    ids = S.tokens(name, 640, 11)
    want = S.oracle_logits(name, p, ids)
    S.close(run(e, ids, [20] + [1] * 620), want, dtype)


@pytest.mark.parametrize("name", ["even", "diff_even"])
def test_graphs_and_eager_steps_agree(name):
    a, _ = S.engine(name, "bfloat16")
    b, _ = S.engine(name, "bfloat16", graphs=False)
    ids = S.tokens(name, 80, 3)
    x, y = run(a, ids, [60] + [1] * 20), run(b, ids, [60] + [1] * 20)
    assert a._graphs and not b._graphs
    # the split of the context follows the context class of the graph, so only rounding may differ
    assert float((x - y).abs().max()) < 1e-2 * float(y.std())


def test_steps_are_checked():
    e, _ = S.engine("only_delta", slots=2, capacity=20)
    s = e.open()
    for bad in (lambda: e.step([s], [[99]]), lambda: e.step([s], [[-1]]), lambda: e.step([s, s], [[1], [2]]), lambda: e.step([1], [[1]]),
                lambda: e.step([s], [[]]), lambda: e.feed(s, [1] * 21), lambda: e.step([s], [[1, 2]], [2]), lambda: e.close(1)):
        with pytest.raises(ValueError):
            bad()
    e.open()
    with pytest.raises(RuntimeError):
        e.open()
    e.feed(s, [1] * 20)
    with pytest.raises(ValueError):
        e.step([s], [[1]])


def greedy(name, params, prompt, n):
    from oracle.layer_stack import decoder
    d, new = decoder(S.CONFIGS[name], params), []
    logits = d.feed(prompt)[-1]
    for _ in range(n):
        new.append(int(np.argmax(logits)))
        logits = d.feed([new[-1]])[-1]
    return new


@pytest.mark.parametrize("name", ["odd", "even", "diff_odd", "diff_even"])
def test_greedy_generation_through_the_scheduler(name):
    """Five prompts over three slots, in fp32: the token ids of the oracle."""
    from reimagined_b200.generate import generate
    e, p = S.engine(name)
    prompts = [S.tokens(name, n, n) for n in (4, 61, 1, 17, 130)]
    assert generate(e, prompts, 15) == [greedy(name, p, ids, 15) for ids in prompts]
    assert len(e._free) == 3


def save_model(folder, name):
    from reimagined_b200.checkpoint import write_safetensors
    w, p = S.weights(name)
    (folder / "config.json").write_text(json.dumps(S.CONFIGS[name]))
    write_safetensors(str(folder / "model.safetensors"), w)
    return p


@pytest.mark.parametrize("name", ["even", "diff_even"])
def test_generation_from_the_command_line(tmp_path, name):
    p = save_model(tmp_path, name)
    prompts = [[3, 200, 17], [9]]
    r = subprocess.run([sys.executable, "-m", "reimagined_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--tokens", "5",
                        *sum((["--prompt", ",".join(map(str, ids))] for ids in prompts), [])], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = [json.loads(x) for x in r.stdout.splitlines() if x.startswith("{")]
    assert got == [{"prompt": ids, "tokens": greedy(name, p, ids, 5)} for ids in prompts]


@pytest.mark.parametrize("name", ["odd", "diff_odd"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(tmp_path, name, dtype):
    model, out = tmp_path / "m", tmp_path / "o"
    model.mkdir()
    out.mkdir()
    p = save_model(model, name)
    a, b = S.tokens(name, 40, 1), S.tokens(name, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[32:], "want": [7, 2]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [8]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"],
                       input="".join(json.dumps(s) + "\n" for s in steps), cwd=str(tmp_path), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = S.oracle_logits(name, p, a), S.oracle_logits(name, p, b)
    for step, want in ((0, la[[0, 29]]), (2, la[[39, 34]]), (3, lb[[8]])):
        S.close(np.fromfile(out / f"{step}.f32", "<f4").reshape(len(want), -1), want, dtype)
    assert not (out / "1.f32").exists()


def test_the_hybrid_generates_through_the_same_entry_point(tbl):
    """The registry's other model: greedy tokens equal those of its engine stepped by hand."""
    from reimagined_b200.decode import DecodeEngine, DecodeSession, synthetic_params
    from reimagined_b200.generate import generate
    cfg = dict(num_layers=2, d_model=128, vocab_size=64, n_heads=2, n_kv_heads=2, mamba_d_state=16, mamba_expand=2, mamba_conv_kernel=4,
               mamba_head_dim=64, mamba_n_groups=1, attention_period=2, attention_slot=1)
    params = synthetic_params(cfg, 5, rope_positions=64)
    prompts = [[3, 9, 4], [60]]
    got = generate(DecodeSession(params, 32), prompts, 6)
    for ids, new in zip(prompts, got):
        e = DecodeEngine(params, batch=1, capacity=32)
        seq = list(ids)
        for i in range(len(ids) + 5):
            logits = e.step([seq[i]])
            if i >= len(ids) - 1:
                seq.append(int(logits.argmax()))
        assert seq[len(ids):] == new
