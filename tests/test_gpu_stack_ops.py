"""The layer-stack operators one by one, through the C ABI, against the plain float64 oracle."""
import ctypes as C

import numpy as np
import pytest

import stack_helpers as S
from oracle import layer_stack as O

pytestmark = pytest.mark.gpu

SIMT, GEMV, TENSOR, ROWS = 1, 2, 3, 4
DELTA_SCAN, DELTA_STEP = 1, 2
CACHE_SIMT, CACHE_TENSOR, EXPANDED = 1, 2, 3


def f64(t):
    return t.detach().float().cpu().numpy().astype(np.float64)


def stream(torch):
    return torch.cuda.current_stream().cuda_stream


def act(torch, a, precision):
    return torch.as_tensor(np.asarray(a, np.float32)).cuda().to(torch.bfloat16 if precision else torch.float32)


class Buf:
    """Keeps tensors alive and hands out pointers."""

    def __init__(self, torch):
        self.torch, self.keep = torch, []

    def f32(self, a):
        self.keep.append(self.torch.as_tensor(np.asarray(a, np.float32)).cuda().contiguous())
        return self.keep[-1].data_ptr()

    def i32(self, a):
        self.keep.append(self.torch.as_tensor(np.asarray(a, np.int32)).cuda())
        return self.keep[-1].data_ptr()

    def view(self, w, bias=None):
        from reimagined_b200 import capi
        self.keep.append(w.cuda().contiguous())
        return capi.DenseView(self.keep[-1].data_ptr(), None if bias is None else self.f32(bias), w.shape[1], w.shape[0])


def assert_close(got, want, rel, what=""):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    err = np.abs(got - want).max() / np.abs(want).max()
    assert np.isfinite(got).all() and err <= rel, f"{what}: {err:.3g}"


# ---- linear layers ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("route,precision", [(SIMT, 0), (SIMT, 1), (GEMV, 0), (GEMV, 1), (TENSOR, 1), (ROWS, 1), (0, 0), (0, 1)])
@pytest.mark.parametrize("m,k,n", [(1, 64, 40), (8, 2048, 48), (13, 200, 100), (27, 4104, 33), (64, 264, 38000), (3, 200, 77), (4, 1032, 5000), (2, 36, 9), (1, 37, 19), (5, 24, 8), (70, 72, 130), (129, 520, 257),
                                   (300, 264, 700)])
def test_dense(cuda, stack_lib, route, precision, m, k, n):
    torch, rng = cuda, np.random.default_rng(m * k + n)
    b = Buf(torch)
    w = torch.as_tensor(rng.standard_normal((n, k)), dtype=torch.float32).bfloat16()
    bias, res = rng.standard_normal(n), rng.standard_normal((m, n)).astype(np.float32)
    ldx = k + (8 if precision else 3)
    x = act(torch, rng.standard_normal((m, ldx)), precision)
    for with_extras in (False, True):
        v = b.view(w, bias if with_extras else None)
        out = torch.full((m, n), float("nan"), device="cuda")
        rc = stack_lib.tbl_dense_forward(C.byref(v), precision, route, x.data_ptr(), ldx, m, b.f32(res) if with_extras else None,
                                         out.data_ptr(), stream(torch))
        if (route == GEMV and (m > 4 or (k % 4 and m > 1))) or (route in (TENSOR, ROWS) and k % 8):
            assert rc == -2
            return
        assert rc == 0
        want = O.linear(f64(x)[:, :k], f64(w), bias if with_extras else None) + (res if with_extras else 0.0)
        # (the tensor cores' fp32 accumulators drop the bits they shift out, which adds up with K)
        assert_close(f64(out), want, 1e-5 if precision else 3e-6, "dense")


def test_dense_tall_tiles_and_the_residual_in_place(cuda, stack_lib):
    torch = cuda
    torch.manual_seed(0)
    b = Buf(torch)
    m, k, n = 3000, 2056, 3400                   # more than a wave of 256 x 256 tiles, ragged in every direction
    w, x = torch.randn(n, k).bfloat16(), torch.randn(m, k).bfloat16().cuda()
    out = torch.randn(m, n, device="cuda")
    want = out.double() + x.double() @ w.cuda().double().T
    assert stack_lib.tbl_dense_forward(C.byref(b.view(w)), 1, TENSOR, x.data_ptr(), k, m, out.data_ptr(), out.data_ptr(), stream(torch)) == 0
    assert float((out.double() - want).abs().max() / want.abs().max()) < 1e-5


@pytest.mark.parametrize("route,precision", [(SIMT, 0), (GEMV, 0), (GEMV, 1), (SIMT, 1), (TENSOR, 1), (ROWS, 1)])
@pytest.mark.parametrize("m,k,ff", [(9, 512, 70), (1, 64, 32), (3, 40, 37), (4, 128, 200), (1, 1024, 3000), (150, 72, 100), (260, 136, 333)])
def test_gated_dense(cuda, stack_lib, route, precision, m, k, ff):
    from reimagined_b200.stack import StackEngine
    torch, rng = cuda, np.random.default_rng(ff)
    if route == GEMV and m > 4:
        return
    b = Buf(torch)
    gate, up = (torch.as_tensor(rng.standard_normal((ff, k)) * k ** -0.5, dtype=torch.float32).bfloat16() for _ in range(2))
    gb, ub = (torch.as_tensor(rng.standard_normal(ff), dtype=torch.float32) for _ in range(2))
    v = b.view(StackEngine._paired(None, gate, up), StackEngine._paired(None, gb, ub).cpu())
    x = act(torch, rng.standard_normal((m, k)), precision)
    out = torch.zeros((m, ff), device="cuda", dtype=x.dtype)
    assert stack_lib.tbl_gated_dense_forward(C.byref(v), precision, route, x.data_ptr(), k, m, ff, out.data_ptr(), stream(torch)) == 0
    want = O.silu(O.linear(f64(x), f64(gate), gb.numpy())) * O.linear(f64(x), f64(up), ub.numpy())
    assert_close(f64(out), want, 4e-3 if precision else 3e-6)


# ---- norm and depth average -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("precision", [0, 1])
@pytest.mark.parametrize("rows,width,count", [(1, 512, 1), (3, 1000, 12), (40, 90, 5), (2, 4100, 19), (33, 516, 9)])
def test_depth_norm(cuda, stack_lib, precision, rows, width, count):
    torch, rng = cuda, np.random.default_rng(width)
    b = Buf(torch)
    src = rows + 4
    hist = rng.standard_normal((count, src, width)).astype(np.float32)
    wts, norm = rng.standard_normal(count), rng.standard_normal(width)
    index = rng.permutation(src)[:rows]
    for weights, idx, eps in ((wts, None, 1e-6), (None, None, 0.5), (wts, index, 0.5)):
        x = torch.full((rows, width), float("nan"), device="cuda")
        h = torch.zeros((rows, width), device="cuda", dtype=torch.bfloat16 if precision else torch.float32)
        rc = stack_lib.tbl_depth_norm(b.f32(hist), src * width, count, None if weights is None else b.f32(weights), precision,
                                      None if idx is None else b.i32(idx), rows, width, eps, b.f32(norm), x.data_ptr(), h.data_ptr(), stream(torch))
        assert rc == 0
        want = O.depth_average(weights, hist) if weights is not None else hist[-1]
        want = np.asarray(want, np.float64)[idx if idx is not None else slice(0, rows)]
        assert_close(f64(x), want, 2e-6)
        assert_close(f64(h), O.rms_norm(want, norm, eps), 4e-3 if precision else 2e-6)


# ---- delta rule -------------------------------------------------------------------------------------------------------------
def delta_mixer(torch, b, heads, dim, rank, rng):
    from reimagined_b200 import capi
    from reimagined_b200.stack import DECAY_RATE, KEY_EPS
    hd, width = heads * dim, 8
    m = capi.DeltaMixer()
    m.in_ = capi.DenseView(b.view(torch.zeros(1, 8).bfloat16()).weight, b.f32(np.zeros(1)), width, 5 * hd + rank)
    w2 = torch.as_tensor(rng.standard_normal((hd, rank)), dtype=torch.float32).bfloat16()
    w0, norm = rng.standard_normal(hd), rng.standard_normal(hd)
    m.decay_up, m.out = b.view(w2, w0), capi.DenseView(b.view(torch.zeros(1, 8).bfloat16()).weight, None, hd, width)
    m.norm, m.heads, m.dim, m.rank, m.decay_rate, m.key_eps = b.f32(norm), heads, dim, rank, DECAY_RATE, KEY_EPS
    return m, f64(w2), np.float32(w0).astype(np.float64), np.float32(norm).astype(np.float64)


def delta_oracle(proj, heads, dim, w2, w0, norm, eps, states):
    """proj [T, ...] of one sequence; states [heads, key, value] updated in place."""
    hd = heads * dim
    r, k, v, g, a = (proj[:, i * hd:(i + 1) * hd].reshape(-1, heads, dim) for i in range(5))
    w = np.exp(-np.exp(-0.5) * O.sigmoid(np.tanh(proj[:, 5 * hd:]) @ w2.T + w0)).reshape(-1, heads, dim)
    out = np.zeros((len(proj), heads, dim))
    for t in range(len(proj)):
        for h in range(heads):
            states[h], out[t, h] = O.delta_step(states[h], r[t, h], k[t, h], v[t, h], w[t, h], O.sigmoid(a[t, h]))
    return O.rms_norm(out, None, eps).reshape(-1, hd) * norm * O.sigmoid(g.reshape(-1, hd))


@pytest.mark.parametrize("precision", [0, 1])
@pytest.mark.parametrize("heads,dim,rank", [(2, 32, 16), (3, 20, 5), (1, 64, 8), (2, 50, 24), (2, 128, 32), (1, 7, 1), (1, 200, 40), (1, 256, 64)])
def test_delta_rule_across_scan_and_single_steps(cuda, stack_lib, precision, heads, dim, rank):
    """Two sequences on slots 2 and 0: a scan, single tokens, and a scan again from the carried states."""
    torch, rng = cuda, np.random.default_rng(dim)
    b = Buf(torch)
    m, w2, w0, norm = delta_mixer(torch, b, heads, dim, rank, rng)
    hd, slots, eps = heads * dim, [2, 0], 1e-3
    states = torch.zeros((3, heads, dim, dim), device="cuda")
    want_states = {s: np.zeros((heads, dim, dim)) for s in slots}
    tol = 1e-2 if precision else 2e-5
    for route, n in ((DELTA_SCAN, 35), (DELTA_STEP, 1), (0, 1), (DELTA_SCAN, 1), (0, 2), (DELTA_SCAN, 17)):
        proj = (0.8 * rng.standard_normal((2 * n, 5 * hd + rank))).astype(np.float32)
        pd = torch.as_tensor(proj).cuda()
        out = torch.zeros((2 * n, hd), device="cuda", dtype=torch.bfloat16 if precision else torch.float32)
        size = stack_lib.tbl_delta_workspace_bytes(C.byref(m), precision, 2 * n)
        ws = torch.empty(size, dtype=torch.uint8, device="cuda")
        rc = stack_lib.tbl_delta_forward(C.byref(m), precision, route, eps, pd.data_ptr(), states.data_ptr(), b.i32(slots), 2, n, out.data_ptr(),
                                         ws.data_ptr(), size, stream(torch))
        assert rc == 0
        for i, s in enumerate(slots):
            want = delta_oracle(proj[i * n:(i + 1) * n].astype(np.float64), heads, dim, w2, w0, norm, eps, want_states[s])
            assert_close(f64(out)[i * n:(i + 1) * n], want, tol, f"n {n} sequence {i}")
            assert_close(f64(states[s]).transpose(0, 2, 1), want_states[s], tol, "state")
    assert not states[1].any()                    # nobody touched the third slot


def test_delta_rule_forgets_and_remembers(cuda, stack_lib):
    """Slow decay and no removal keep the first token for 400 tokens; a removal rate of one wipes its direction."""
    torch, rng = cuda, np.random.default_rng(1)
    b = Buf(torch)
    dim, n = 32, 400
    m, w2, w0, norm = delta_mixer(torch, b, 1, dim, 4, rng)
    slow = np.full(dim, -9.0)
    m.decay_up.bias = b.f32(slow)
    proj = np.zeros((n, 5 * dim + 4), np.float32)
    key = rng.standard_normal(dim).astype(np.float32)
    proj[0, dim:2 * dim] = key
    proj[0, 2 * dim:3 * dim] = rng.standard_normal(dim)
    proj[:, :dim] = key                            # every token reads with the first token's key
    proj[:, 4 * dim:5 * dim] = -20.0
    for wipe in (False, True):
        if wipe:
            proj[200, dim:2 * dim] = key
            proj[200, 4 * dim:5 * dim] = 20.0
        states = torch.zeros((1, 1, dim, dim), device="cuda")
        out = torch.zeros((n, dim), device="cuda")
        size = stack_lib.tbl_delta_workspace_bytes(C.byref(m), 0, n)
        ws = torch.empty(size, dtype=torch.uint8, device="cuda")
        assert stack_lib.tbl_delta_forward(C.byref(m), 0, 0, 1e-2, torch.as_tensor(proj).cuda().data_ptr(), states.data_ptr(), b.i32([0]), 1, n,
                                           out.data_ptr(), ws.data_ptr(), size, stream(torch)) == 0
        want = delta_oracle(proj.astype(np.float64), 1, dim, w2, slow, norm, 1e-2, np.zeros((1, dim, dim)))
        assert_close(f64(out), want, 1e-4)
        assert (np.abs(want[300]).max() < 0.05 * np.abs(want[100]).max()) == wipe


# ---- latent attention ---------------------------------------------------------------------------------------------------------
class Latent:
    """A latent-attention mixer with random weights, its cache, and the same in the oracle."""

    def __init__(self, torch, lib, cfg, precision, slots=3, capacity=420, seed=0, eps=1e-4):
        from reimagined_b200 import capi
        self.torch, self.lib, self.cfg, self.precision, self.capacity, self.eps = torch, lib, cfg, precision, capacity, eps
        rng = self.rng = np.random.default_rng(seed)
        self.b = b = Buf(torch)
        H, d, rd, vd, q, R = (cfg[n] for n in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
        w = lambda n, k: torch.as_tensor(rng.standard_normal((n, k)) * k ** -0.5, dtype=torch.float32).bfloat16()
        uq, uk, uv = w(H * (d + rd), q), w(H * d, R), w(H * vd, R)
        qn, kn = rng.uniform(0.5, 1.5, q), rng.uniform(0.5, 1.5, R)
        self.P = {"dq.norm": np.float32(qn), "dkv.norm": np.float32(kn), "uq": f64(uq), "uk": f64(uk), "uv": f64(uv)}
        m = self.m = capi.LatentMixer()
        dummy = b.view(torch.zeros(1, 8).bfloat16()).weight
        self.cols = q + R + rd + H * vd
        m.in_, m.out = capi.DenseView(dummy, None, 8, self.cols), capi.DenseView(dummy, None, H * vd, 8)
        m.uq, m.uk, m.uv = b.view(uq), b.view(uk), b.view(uv)
        m.uk_t = b.view(uk.reshape(H, d, R).transpose(1, 2).reshape(H * R, d)).weight
        m.q_norm, m.kv_norm = b.f32(qn), b.f32(kn)
        ang = np.arange(capacity)[:, None] * cfg["rot"]["base"] ** (-2.0 * np.arange(rd // 2) / rd)
        m.rope_cos, m.rope_sin, m.rope_positions = b.f32(np.cos(ang)), b.f32(np.sin(ang)), capacity
        m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale = H, d, rd, vd, q, R, cfg["scale"]
        cw = (R + rd + 7) // 8 * 8
        self.cache = torch.zeros((slots, capacity, cw), device="cuda", dtype=torch.bfloat16 if precision else torch.float32)
        self.positions = torch.zeros(slots, dtype=torch.int32, device="cuda")
        self.ocache = {}

    def forward(self, route, slots, proj, check_rc=0):
        torch, n_seq = self.torch, len(slots)
        n = len(proj) // n_seq
        context = int(self.positions[slots].max()) + n
        H, vd = self.cfg["heads"], self.cfg["vdim"]
        out = torch.zeros((n_seq * n, H * vd), device="cuda", dtype=self.cache.dtype)
        size = self.lib.tbl_latent_workspace_bytes(C.byref(self.m), self.precision, n_seq, n, context)
        ws = torch.full((size,), 255, dtype=torch.uint8, device="cuda")          # NaN patterns: nothing unwritten may be used
        pd = torch.as_tensor(np.asarray(proj, np.float32)).cuda()
        rc = self.lib.tbl_latent_forward(C.byref(self.m), self.precision, route, self.eps, pd.data_ptr(), self.cache.data_ptr(), self.capacity,
                                         self.b.i32(slots), self.positions.data_ptr(), n_seq, n, context, out.data_ptr(), ws.data_ptr(), size,
                                         stream(torch))
        assert rc == check_rc
        if rc == 0:
            self.positions[slots] += n
        return f64(out)

    def oracle(self, slots, proj):
        """The oracle's mixer reads h; identity projections turn the stacked products into that."""
        c, H, vd = self.cfg, self.cfg["heads"], self.cfg["vdim"]
        q, R, rd = c["q_rank"], c["kv_rank"], c["rot_dim"]
        eye = np.eye(self.cols)
        P = {**self.P, "dq": eye[:q], "dkv": eye[q:q + R + rd], "g": eye[q + R + rd:], "o": np.eye(H * vd)}
        n = len(proj) // len(slots)
        return np.concatenate([O.latent_attention(np.asarray(proj[i * n:(i + 1) * n], np.float64), P, "", c, self.eps, self.ocache.setdefault(s, []))
                               for i, s in enumerate(slots)])


SIZES = {
    "odd": S.latent(5, 20, 12, 28, 36, 44, 0.8, 90.0)["mixer"],
    "tiny": S.latent(2, 3, 2, 5, 7, 9, 1.5, 7.0)["mixer"],
    "small": S.latent(3, 48, 16, 80, 64, 80, 0.6, 1e4)["mixer"],
    "heads20": S.latent(20, 80, 32, 16, 40, 192, 0.35, 300.0)["mixer"],
    "heads40": S.latent(40, 16, 16, 32, 24, 128, 0.9, 300.0)["mixer"],
    "wide": S.latent(2, 128, 64, 128, 128, 512, 0.3, 2e3)["mixer"],
    "latent500": S.latent(2, 30, 10, 20, 16, 490, 0.5, 2e3)["mixer"],
    "latent1000": S.latent(1, 16, 16, 16, 16, 1000, 0.5, 2e3)["mixer"],
}
ROUTES = {CACHE_SIMT: list(SIZES), CACHE_TENSOR: ["small", "heads20", "heads40", "wide"], EXPANDED: ["small", "heads20", "heads40", "wide"]}


@pytest.mark.parametrize("precision,route,size", [(0, CACHE_SIMT, s) for s in ROUTES[CACHE_SIMT]] +
                         [(1, r, s) for r in ROUTES for s in ROUTES[r]] + [(0, 0, "small"), (1, 0, "small"), (1, 0, "odd")])
def test_latent_attention(cuda, stack_lib, precision, route, size):
    """A prompt in portions (two tokens among them), then single tokens, on two slots at different places."""
    a = Latent(cuda, stack_lib, SIZES[size], precision)
    rng, tol = np.random.default_rng(5), 3e-2 if precision else 2e-5
    steps = [([1], 130), ([1], 2), ([2], 61), ([1, 2], 3), ([1, 2], 1), ([2, 1], 1), ([1, 2], 140), ([2], 1)]
    for slots, n in steps:
        proj = rng.standard_normal((len(slots) * n, a.cols)).astype(np.float32)
        got, want = a.forward(route, slots, proj), a.oracle(slots, proj)
        assert_close(got, want, tol, f"slots {slots} n {n}")
        err = np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean())
        assert err.max() < tol, (slots, n, int(err.argmax()), err.max())


@pytest.mark.parametrize("route,size", [(CACHE_TENSOR, "odd"), (EXPANDED, "odd"), (CACHE_TENSOR, "latent500"), (EXPANDED, "latent1000")])
def test_latent_routes_refuse_sizes_they_do_not_take(cuda, stack_lib, route, size):
    a = Latent(cuda, stack_lib, SIZES[size], 1)
    a.forward(route, [0], np.zeros((2, a.cols)), check_rc=-2) if not (route == EXPANDED and size == "latent1000") else None
    a.precision = 0
    a.forward(route, [0], np.zeros((2, a.cols)), check_rc=-2)


@pytest.mark.parametrize("precision,route,size", [(0, CACHE_SIMT, "small"), (1, CACHE_SIMT, "small"), (1, CACHE_TENSOR, "small"), (1, EXPANDED, "small"),
                                                  (1, CACHE_TENSOR, "heads20"), (1, EXPANDED, "wide")])
def test_latent_attention_finds_one_key(cuda, stack_lib, precision, route, size):
    """Queries aimed at a single cached token: the first ones, both sides of tile and block borders, the latest, itself.  A
    key that is missing or off by one replaces the whole output."""
    cfg = dict(SIZES[size])
    a = Latent(cuda, stack_lib, cfg, precision, seed=2)
    rng, n = np.random.default_rng(6), 390
    H, d, rd, q, R = (cfg[k] for k in ("heads", "dim", "rot_dim", "q_rank", "kv_rank"))
    proj = rng.standard_normal((n, a.cols)).astype(np.float32)
    proj[:, q + R:q + R + rd] *= 0.02              # the rotated part stays out of the way
    lat = O.rms_norm(proj[:, q:q + R], a.P["dkv.norm"], a.eps)
    head = H - 1
    uq = a.P["uq"].reshape(H, d + rd, q)[head, :d]
    uk = a.P["uk"].reshape(H, d, R)[head]
    borders = [0, 1, 2, 63, 64, 65, 126, 127, 128, 129, 191, 192, 255, 256, 257, 383, 384]
    target = np.array([borders[t % len(borders)] if borders[t % len(borders)] <= t else t for t in range(n)])
    target[::7] = np.arange(n)[::7]                # itself
    target[3::11] = np.maximum(np.arange(n)[3::11] - 1, 0)
    proj[:, :q] = (lat[target] @ uk.T @ uq) / a.P["dq.norm"]
    # scale so that the target's score is 40 on average (the others: noise of a few units)
    cq = O.rms_norm(proj[:, :q], a.P["dq.norm"], a.eps)
    own = np.einsum("tr,tr->t", cq @ uq.T @ uk, lat[target])
    cfg["scale"] = a.m.scale = float(40.0 / own.mean())
    got = np.concatenate([a.forward(route, [0], proj[:300]), a.forward(route, [0], proj[300:389]), a.forward(route if route != EXPANDED else 0, [0], proj[389:])])
    want = a.oracle([0], proj)
    vd = cfg["vdim"]
    value = (lat @ a.P["uv"].reshape(H, vd, R)[head].T)[target] * O.sigmoid(proj[:, -vd:])
    w = want[:, head * vd:]
    assert np.median(np.abs(w - value).max(axis=1) / np.abs(value).max(axis=1)) < 0.05          # the construction works
    g = got[:, head * vd:]
    err = np.sqrt(((g - w) ** 2).mean(axis=1) / (w ** 2).mean(axis=1))
    assert err.max() < (0.1 if precision else 1e-4), (int(err.argmax()), err.max())


def test_latent_attention_reports_a_full_cache(cuda, stack_lib):
    a = Latent(cuda, stack_lib, SIZES["small"], 1, capacity=16)
    stack_lib.tbl_device_status(stream(cuda))
    a.forward(0, [0], np.zeros((10, a.cols)))
    assert stack_lib.tbl_device_status(stream(cuda)) == 0
    a.positions[0] = 15                             # the step's context claims less than the device holds
    size = stack_lib.tbl_latent_workspace_bytes(C.byref(a.m), 1, 1, 2, 16)
    ws, pd = cuda.empty(size, dtype=cuda.uint8, device="cuda"), cuda.zeros((2, a.cols), device="cuda")
    out = cuda.zeros((2, 3 * 80), device="cuda", dtype=cuda.bfloat16)
    before = a.cache[1:].clone()
    assert stack_lib.tbl_latent_forward(C.byref(a.m), 1, 0, 1e-4, pd.data_ptr(), a.cache.data_ptr(), 16, a.b.i32([0]), a.positions.data_ptr(), 1, 2, 16,
                                        out.data_ptr(), ws.data_ptr(), size, stream(cuda)) == 0
    assert stack_lib.tbl_device_status(stream(cuda)) == 4
    assert cuda.equal(before, a.cache[1:])


# ---- residual streams and Dynamic Tanh ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("precision", [0, 1])
@pytest.mark.parametrize("rows,width,streams", [(1, 512, 2), (3, 1000, 1), (40, 90, 3), (2, 4100, 4), (33, 516, 8), (5, 37, 5), (70, 64, 6), (32, 2048, 7)])
def test_stream_norm(cuda, stack_lib, precision, rows, width, streams):
    """Update, store, sum, next input and both norms; then rows picked out without a store."""
    torch, rng = cuda, np.random.default_rng(width)
    b = Buf(torch)
    xs, y = rng.standard_normal((streams, rows, width)).astype(np.float32), rng.standard_normal((rows, width)).astype(np.float32)
    mix, out_w, in_w = rng.standard_normal((streams, streams)), rng.standard_normal(streams), rng.standard_normal(streams)
    norm, bias, alpha, eps = rng.standard_normal(width), rng.standard_normal(width), 0.7, 0.3
    index = rng.integers(0, rows, max(1, rows // 2))
    tol = 4e-3 if precision else 2e-6
    for kind in (0, 1):
        for update, store, weights, idx in ((True, 1, in_w, None), (False, 0, in_w, None), (True, 0, None, index), (True, 0, in_w, None)):
            n = rows if idx is None else len(idx)
            x = torch.as_tensor(xs).cuda()
            total = torch.full((n, width), float("nan"), device="cuda")
            h = torch.zeros((n, width), device="cuda", dtype=torch.bfloat16 if precision else torch.float32)
            rc = stack_lib.tbl_stream_norm(x.data_ptr(), rows * width, streams, b.f32(y) if update else None, b.f32(mix), b.f32(out_w), store,
                                           None if weights is None else b.f32(weights), precision, None if idx is None else b.i32(idx), n, width, kind,
                                           eps, alpha, b.f32(norm), b.f32(bias), total.data_ptr(), h.data_ptr(), stream(torch))
            assert rc == 0
            f32 = lambda a: np.float32(a).astype(np.float64)
            new = O.streams_out(list(xs.astype(np.float64)), f32(mix), f32(out_w), y) if update else list(xs.astype(np.float64))
            pick = slice(None) if idx is None else idx
            assert_close(f64(total), sum(new)[pick], 3e-6, "sum")
            u = O.streams_in(new, np.ones(streams) if weights is None else f32(weights))[pick]
            want = O.rms_norm(u, f32(norm), eps) if kind == 0 else O.dynamic_tanh(u, np.float32(alpha), f32(norm), f32(bias))
            assert_close(f64(h), want, tol, "h")
            for got, a in zip(f64(x), new if store else xs):
                assert_close(got, a, 3e-6 if store else 0, "streams")


@pytest.mark.parametrize("route,precision", [(SIMT, 0), (GEMV, 0), (GEMV, 1), (SIMT, 1), (TENSOR, 1), (ROWS, 1)])
@pytest.mark.parametrize("m,k,ff", [(9, 512, 70), (1, 64, 32), (3, 40, 37), (150, 72, 100)])
def test_gated_dense_with_gelu(cuda, stack_lib, route, precision, m, k, ff):
    from reimagined_b200.stack import StackEngine
    torch, rng = cuda, np.random.default_rng(ff + 1)
    if route == GEMV and m > 4:
        return
    b = Buf(torch)
    gate, up = (torch.as_tensor(2.0 * rng.standard_normal((ff, k)) * k ** -0.5, dtype=torch.float32).bfloat16() for _ in range(2))
    v = b.view(StackEngine._paired(None, gate, up))
    x = act(torch, rng.standard_normal((m, k)), precision)
    out = torch.zeros((m, ff), device="cuda", dtype=x.dtype)
    assert stack_lib.tbl_gated_dense_act_forward(C.byref(v), precision, route, 1, x.data_ptr(), k, m, ff, out.data_ptr(), stream(torch)) == 0
    want = O.gelu_tanh(O.linear(f64(x), f64(gate))) * O.linear(f64(x), f64(up))
    assert_close(f64(out), want, 4e-3 if precision else 3e-6)


# ---- attention with grouped heads and one or two maps ---------------------------------------------------------------------------
A_SIMT, A_STREAM, A_FLASH = 1, 2, 3


class Attention:
    """An attention mixer on given projections, its cache, and the same in the oracle."""

    def __init__(self, torch, lib, cfg, precision, slots=3, capacity=420, eps=1e-2, lam=0.6, gated=True, owner=None):
        from reimagined_b200 import capi
        self.torch, self.lib, self.cfg, self.precision, self.capacity, self.eps, self.gated = torch, lib, cfg, precision, capacity, eps, gated
        self.b, self.owner, self.n_slots = Buf(torch), owner, slots
        H, G, d, vd = (cfg[n] for n in ("heads", "kv_heads", "dim", "vdim"))
        self.maps = maps = 2 if "diff" in cfg else 1
        self.sizes = [("q", H * maps * d)] + ([("k", G * maps * d), ("v", G * vd)] if owner is None else []) + ([("g", H * vd)] if gated else [])
        self.cols = sum(n for _, n in self.sizes)
        dummy = self.b.view(torch.zeros(1, 8).bfloat16()).weight
        m = self.m = capi.AttentionMixer()
        m.in_, m.out = capi.DenseView(dummy, None, 8, self.cols), capi.DenseView(dummy, None, H * vd, 8)
        m.heads, m.kv_heads, m.dim, m.vdim, m.maps, m.gated, m.kv_from, m.scale = H, G, d, vd, maps, int(gated), -1 if owner is None else 0, cfg["scale"]
        m.lambda_, m.out_scale = lam, 1.0 - cfg.get("diff", 0.0)
        # lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
        self.P = {n: np.eye(d)[0] for n in ("lq1", "lk1", "lk2")}
        self.P["lq2"] = np.eye(d)[0] * np.log(np.e - lam + cfg.get("diff", 0.0))
        if "q_temp" in cfg:
            m.temperature = self.b.f32(O.query_temperature(np.arange(capacity), cfg["q_temp"]["coef"], cfg["q_temp"]["every"]))
            m.temperature_positions = capacity
        cw = lib.tbl_attention_cache_width(C.byref(m))
        dtype = torch.bfloat16 if precision else torch.float32
        self.cache = torch.zeros((slots, G, capacity, cw), device="cuda", dtype=dtype) if owner is None else owner.cache
        self.positions = torch.zeros(slots, dtype=torch.int32, device="cuda") if owner is None else owner.positions
        self.ocache = {} if owner is None else owner.ocache

    def forward(self, route, slots, proj, check_rc=0, advance=True):
        torch, n_seq = self.torch, len(slots)
        n = len(proj) // n_seq
        context = int(self.positions[slots].max()) + n
        out = torch.zeros((n_seq * n, self.cfg["heads"] * self.cfg["vdim"]), device="cuda", dtype=self.cache.dtype)
        size = self.lib.tbl_attention_workspace_bytes(C.byref(self.m), self.precision, n_seq, n, context)
        ws = torch.full((size,), 255, dtype=torch.uint8, device="cuda")          # NaN patterns: nothing unwritten may be used
        pd = torch.as_tensor(np.asarray(proj, np.float32)).cuda()
        rc = self.lib.tbl_attention_forward(C.byref(self.m), self.precision, route, self.eps, pd.data_ptr(), self.cache.data_ptr(), self.n_slots,
                                            self.capacity, self.b.i32(slots), self.positions.data_ptr(), n_seq, n, context, out.data_ptr(),
                                            ws.data_ptr(), size, stream(torch))
        assert rc == check_rc
        if rc == 0 and advance:
            self.positions[slots] += n
        return f64(out)

    def oracle(self, slots, proj):
        """The oracle's mixer reads h; identity projections turn the stacked products into that."""
        eye, at, P = np.eye(self.cols), 0, dict(self.P)
        for name, n in self.sizes:
            P[name], at = eye[at:at + n], at + n
        P["o"] = np.eye(self.cfg["heads"] * self.cfg["vdim"])
        n = len(proj) // len(slots)
        return np.concatenate([O.grouped_attention(np.asarray(proj[i * n:(i + 1) * n], np.float64), P, "", self.cfg, self.eps, self.ocache.setdefault(s, []))
                               for i, s in enumerate(slots)])


def att(*args, diff=True, temp=True):
    m = dict(S.attention(*args)["mixer"])
    for name, keep in (("diff", diff), ("q_temp", temp)):
        if not keep:
            del m[name]
    return m


ATT = {
    "odd": att(6, 3, 10, 28, 0.8, 0.3, 0.5, 7),
    "tiny": att(2, 1, 3, 5, 0.4, 0.0, 0.5, 2),
    "small": att(4, 2, 48, 80, 0.3, 0.6, 0.4, 32),
    "group12": att(12, 1, 16, 32, 0.5, 0.2, 0.3, 100),
    "group20": att(40, 2, 32, 64, 0.3, 0.5, 0.2, 50),
    "wide": att(2, 1, 128, 256, 0.15, 0.4, 0.5, 40),
    "values144": att(3, 3, 24, 144, 0.4, 0.5, 0.4, 64),
    "plain": att(6, 2, 64, 64, 0.2, 0, 0.5, 20, diff=False),
    "plain_odd": att(5, 1, 20, 36, 0.4, 0, 0, 1, diff=False, temp=False),
    "plain_wide": att(2, 2, 192, 200, 0.1, 0, 0, 1, diff=False, temp=False),
    "keys300": att(2, 1, 300, 512, 0.1, 0.3, 0.5, 64),
}
A_ROUTES = {A_SIMT: list(ATT), A_STREAM: [s for s in ATT if s != "keys300"], A_FLASH: [s for s in ATT if s != "keys300"]}


def rows_close(got, want, tol, what):
    """Every row by itself: its error against the rows' usual size."""
    err = np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean())
    assert np.isfinite(got).all() and err.max() < tol, (what, int(err.argmax()), err.max())


@pytest.mark.parametrize("precision,route,size", [(0, A_SIMT, s) for s in ATT] + [(1, r, s) for r in A_ROUTES for s in A_ROUTES[r]] +
                         [(0, 0, "small"), (1, 0, "small"), (1, 0, "odd"), (1, 0, "keys300"), (1, 0, "plain_wide")])
def test_attention(cuda, stack_lib, precision, route, size):
    """A prompt in portions (two tokens among them), then single tokens, on two slots at different places."""
    # (heads of five values come close to zero as a whole: a larger eps, so that their norm does not blow up the rounding)
    a = Attention(cuda, stack_lib, ATT[size], precision, gated=size not in ("plain", "tiny"), eps=0.5 if size == "tiny" else 1e-2)
    rng, tol = np.random.default_rng(5), 3e-2 if precision else 2e-5
    for slots, n in [([1], 130), ([1], 2), ([2], 61), ([1, 2], 3), ([1, 2], 1), ([2, 1], 1), ([1, 2], 140), ([2], 1)]:
        proj = rng.standard_normal((len(slots) * n, a.cols)).astype(np.float32)
        rows_close(a.forward(route, slots, proj), a.oracle(slots, proj), tol, f"slots {slots} n {n}")
    assert not a.cache[0].any()                   # nobody touched the first slot


@pytest.mark.parametrize("precision,route", [(0, A_SIMT), (1, A_SIMT), (1, A_STREAM), (1, A_FLASH)])
def test_attention_over_another_layers_cache(cuda, stack_lib, precision, route):
    """The second mixer has queries, scale, temperature and maps' weights of its own, and leaves the cache alone."""
    first = Attention(cuda, stack_lib, ATT["small"], precision)
    second = Attention(cuda, stack_lib, {**ATT["small"], "scale": 0.5, "diff": 0.1, "q_temp": {"coef": 0.9, "every": 10}}, precision, lam=-0.4, owner=first)
    rng, tol = np.random.default_rng(7), 3e-2 if precision else 2e-5
    for slots, n in [([1], 131), ([2], 2), ([1, 2], 1), ([2, 1], 37)]:
        proj, own = (rng.standard_normal((len(slots) * n, x.cols)).astype(np.float32) for x in (first, second))
        rows_close(first.forward(route, slots, proj, advance=False), first.oracle(slots, proj), tol, "first")
        before = first.cache.clone()
        rows_close(second.forward(route, slots, own), second.oracle(slots, own), tol, "second")
        assert cuda.equal(before, first.cache)


@pytest.mark.parametrize("route,size", [(A_STREAM, "keys300"), (A_FLASH, "keys300")])
def test_attention_routes_refuse_sizes_they_do_not_take(cuda, stack_lib, route, size):
    a = Attention(cuda, stack_lib, ATT[size], 1)
    a.forward(route, [0], np.zeros((2, a.cols)), check_rc=-2)
    a = Attention(cuda, stack_lib, ATT["small"], 0)
    a.forward(route, [0], np.zeros((2, a.cols)), check_rc=-2)


@pytest.mark.parametrize("precision,route,size", [(0, A_SIMT, "odd")] + [(1, r, s) for r in (A_SIMT, A_STREAM, A_FLASH)
                                                                         for s in ("odd", "small", "group12", "wide", "plain")])
@pytest.mark.parametrize("aimed", [0, 1])
def test_attention_finds_one_key(cuda, stack_lib, precision, route, size, aimed):
    """One map's queries aim at a single cached token: the first ones, both sides of tile and block borders, the latest,
    itself.  The other map spreads out.  A key that is missing or off by one replaces the output."""
    cfg = {**ATT[size], "q_temp": {"coef": 0.1, "every": 50}}
    maps = 2 if "diff" in cfg else 1
    if aimed >= maps:
        return
    a = Attention(cuda, stack_lib, cfg, precision, lam=1.5)
    rng, n = np.random.default_rng(6), 400
    H, G, d, vd = (cfg[k] for k in ("heads", "kv_heads", "dim", "vdim"))
    proj = rng.standard_normal((n, a.cols)).astype(np.float32)
    borders = [0, 1, 2, 15, 16, 31, 32, 63, 64, 65, 126, 127, 128, 129, 191, 192, 255, 256, 257, 383, 384]
    target = np.array([borders[t % len(borders)] if borders[t % len(borders)] <= t else t for t in range(n)])
    target[::7] = np.arange(n)[::7]                # itself
    target[3::11] = np.maximum(np.arange(n)[3::11] - 1, 0)
    q = proj[:, :H * maps * d].reshape(n, H, maps, d)
    k = proj[:, H * maps * d:(H + G) * maps * d].reshape(n, G, maps, d)
    k /= np.sqrt((k ** 2).sum(-1, keepdims=True))
    aim = 45.0 / cfg["scale"]                      # the target's score; the others follow from the angle to it
    for h in range(H):
        q[:, h] *= 0.1
        q[:, h, aimed] = aim * k[target, h // (H // G), aimed]
    cuts = [300, 60, 1, 2, 37] if route != A_STREAM else [300] + [1] * 40 + [2, 58]
    got, at = [], 0
    for c in cuts:
        got.append(a.forward(route, [0], proj[at:at + c]))
        at += c
    got, want = np.concatenate(got), a.oracle([0], proj)
    if maps == 1:                                  # the construction works
        v = np.array([e[1] for e in a.ocache[0]])[target].repeat(H // G, axis=1).reshape(n, -1)
        gate = O.sigmoid(proj[:, -H * vd:])
        assert np.median(np.abs(want - v * gate).max(axis=1) / np.abs(v).max(axis=1)) < 0.2
    rows_close(got, want, 6e-2 if precision else 1e-4, "aimed")


def test_attention_does_not_depend_on_what_else_is_in_the_batch_or_on_slots(cuda, stack_lib):
    """The same rows alone, and in other slots beside longer sequences, prompt and decode."""
    rng = np.random.default_rng(8)
    for n, route in ((100, A_FLASH), (1, A_STREAM), (5, A_STREAM)):
        a, b = (Attention(cuda, stack_lib, ATT["small"], 1) for _ in range(2))
        history, other = rng.standard_normal((150, a.cols)), rng.standard_normal((260, a.cols))
        a.forward(A_FLASH, [0], history)
        b.forward(A_FLASH, [1], other)
        b.forward(A_FLASH, [2], history)
        x, y = rng.standard_normal((n, a.cols)), rng.standard_normal((n, a.cols))
        alone, beside = a.forward(route, [0], x), b.forward(route, [1, 2], np.concatenate([y, x]))[n:]
        # the split of the cache may differ: rounding only
        assert np.abs(alone - beside).max() <= (0 if route == A_FLASH else 1e-2) * np.abs(alone).max() + 1e-6


def test_attention_reports_a_full_cache(cuda, stack_lib):
    a = Attention(cuda, stack_lib, ATT["small"], 1, capacity=16)
    stack_lib.tbl_device_status(stream(cuda))
    a.forward(0, [0], np.zeros((10, a.cols)))
    assert stack_lib.tbl_device_status(stream(cuda)) == 0
    for n, pos in ((2, 15), (1, 16)):               # the step's context claims less than the device holds
        a.positions[0] = pos
        size = stack_lib.tbl_attention_workspace_bytes(C.byref(a.m), 1, 1, n, 16)
        ws, pd = cuda.empty(size, dtype=cuda.uint8, device="cuda"), cuda.ones((n, a.cols), device="cuda")
        out = cuda.zeros((n, 4 * 80), device="cuda", dtype=cuda.bfloat16)
        before = a.cache[1:].clone()
        assert stack_lib.tbl_attention_forward(C.byref(a.m), 1, 0, 1e-4, pd.data_ptr(), a.cache.data_ptr(), 3, 16, a.b.i32([0]), a.positions.data_ptr(), 1,
                                               n, 16, out.data_ptr(), ws.data_ptr(), size, stream(cuda)) == 0
        assert stack_lib.tbl_device_status(stream(cuda)) == 4
        assert cuda.equal(before, a.cache[1:])


@pytest.mark.parametrize("precision,route", [(0, A_SIMT), (1, A_STREAM), (1, A_FLASH)])
def test_attention_finds_keys_far_back_in_a_long_cache(cuda, stack_lib, precision, route):
    """More splits of the context than a cluster has: single tokens and a short portion behind a long prompt, the first
    map's queries aimed at keys at its start, at tile and block borders and at its end."""
    cfg = {**ATT["small"], "heads": 2, "kv_heads": 1, "q_temp": {"coef": 0.05, "every": 1000}}
    a = Attention(cuda, stack_lib, cfg, precision, slots=2, capacity=4800, lam=1.2)
    H, d, vd, n = 2, cfg["dim"], cfg["vdim"], 4700
    rng = np.random.default_rng(3)
    proj = rng.standard_normal((n + 28, a.cols)).astype(np.float32)
    k = proj[:, H * 2 * d:(H + 1) * 2 * d].reshape(-1, 2, d)
    k /= np.sqrt((k ** 2).sum(-1, keepdims=True))
    v = proj[:, (H + 1) * 2 * d:(H + 1) * 2 * d + vd]
    target = [0, 1, 63, 64, 127, 128, 2047, 2048, 4095, 4096, 4607, 4608, 4699, 4700] * 2
    q = proj[:, :H * 2 * d].reshape(-1, H, 2, d)
    q *= 0.1
    for i, t in enumerate(target):
        q[n + i, :, 0] = 45.0 / cfg["scale"] * k[t, 0]
    a.forward(0, [1], proj[:n])
    a.ocache[1] = [(k[t][None].astype(np.float64), v[t][None].astype(np.float64)) for t in range(n)]
    at = n
    for c in [1] * 14 + [3, 2, 9]:
        got, want = a.forward(route, [1], proj[at:at + c]), a.oracle([1], proj[at:at + c])
        rows_close(got, want, 6e-2 if precision else 1e-4, at)
        at += c
