"""Tied attention, routing and grouped products one kernel at a time, against float64 statements of the same operator."""
import numpy as np
import pytest
import torch

from oracle import topunex as O

pytestmark = pytest.mark.gpu

DTYPES = {"float32": (torch.float32, 3e-5), "bfloat16": (torch.bfloat16, 1.2e-2)}
PAGE = 64


def _rand(rng, *shape, scale=1.0, dtype=torch.bfloat16):
    """(device tensor, the float64 values it holds)"""
    t = torch.from_numpy((rng.standard_normal(shape) * scale).astype(np.float32)).to(dtype)
    return t.cuda(), t.double().numpy()


def _close(got, want, tol):
    got = got.double().cpu().numpy()
    assert np.isfinite(got).all()
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= tol, err


@pytest.fixture(autouse=True)
def _status():
    yield
    from cacheir_b200 import _lib
    assert _lib.group_device_status() == 0


# ---- dense products: what the paired epilogues, biases and tails add -----------------------------------------------------
@pytest.mark.parametrize("t,n,k", [(1, 8, 8), (17, 136, 264), (64, 512, 2048), (129, 250, 72), (520, 1024, 128)])
def test_dense_products_with_bias_pairs_and_tail(t, n, k):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(t + n)
    x, xn = _rand(rng, t, k)
    w, wn = _rand(rng, n, k, scale=1.5 * k ** -0.5)
    b, bn = _rand(rng, n, dtype=torch.float32)
    y = xn @ wn.T + bn
    out = torch.empty((t, n), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, out, bias=b)
    _close(out, y, 5e-3)
    g, u = y[:, 0::2], y[:, 1::2]
    half = torch.empty((t, n // 2), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, half, epilogue=H.DENSE_SWIGLU, bias=b)
    _close(half, g * O.sigmoid(g) * u, 6e-3)
    tail_cols = min(n - 2, 7 if n > 8 else 3)
    tail_cols -= (n - tail_cols) % 2
    tail = torch.full((t, tail_cols + 2), 5.0, device="cuda")
    pairs = (n - tail_cols) // 2
    H.dense_gemm(x, w, half[:, :pairs], epilogue=H.DENSE_CLAMPED_GLU, limit=0.75, tail=tail[:, :tail_cols])
    z = xn @ wn.T
    g, u = np.minimum(z[:, 0:2 * pairs:2], 0.75), np.clip(z[:, 1:2 * pairs:2], -0.75, 0.75)
    _close(half[:, :pairs], g * O.sigmoid(1.702 * g) * (u + 1), 6e-3)
    _close(tail[:, :tail_cols], z[:, 2 * pairs:], 1e-5)
    assert float((tail[:, tail_cols:] - 5).abs().max()) == 0.0
    f32 = H.dense_simple(x.float(), w.float(), torch.empty((t, n), device="cuda"), bias=b)
    _close(f32, y, 2e-6)
    _close(H.glu_pairs(f32, torch.empty((t, n // 2), device="cuda"), H.DENSE_CLAMPED_GLU, 0.5),
           np.minimum(y[:, 0::2], 0.5) * O.sigmoid(1.702 * np.minimum(y[:, 0::2], 0.5)) * (np.clip(y[:, 1::2], -0.5, 0.5) + 1), 2e-5)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("rows,width", [(1, 1), (3, 90), (40, 2304)])
def test_rms_rows(rows, width, dtype):
    from cacheir_b200 import hybrid_ops as H

    td, _ = DTYPES[dtype]
    rng = np.random.default_rng(width)
    x, xn = _rand(rng, rows, width, dtype=torch.float32)
    w, wn = _rand(rng, width, dtype=torch.float32)
    pick = rng.integers(0, rows, rows + 2).astype(np.int32)
    got = H.rms_rows(x, w, 0.01, torch.empty((rows + 2, width), device="cuda", dtype=td), torch.from_numpy(pick).cuda())
    _close(got, O.rms(xn[pick], 0.01) * wn, 5e-3 if dtype == "bfloat16" else 2e-6)


# ---- routing and experts ---------------------------------------------------------------------------------------------------
def _routing(rows, experts, top, counters=None):
    from cacheir_b200 import expert_ops as X

    def ints(*shape):
        return torch.full(shape, -7, device="cuda", dtype=torch.int32)
    counters = torch.zeros(experts + 1, device="cuda", dtype=torch.int32) if counters is None else counters
    return X.Routing(experts, top, counters, ints(experts + 1), ints(rows * top), ints(rows, top), ints(rows, top),
                     torch.empty((rows, top), device="cuda"))


def _route(rng, rows, experts, top, padding=0, scale=2.5, x=None, placed=None):
    from cacheir_b200 import expert_ops as X

    z, zn = _rand(rng, rows, experts + 3, dtype=torch.float32)
    seg = torch.arange(rows, device="cuda", dtype=torch.int32)
    if padding:
        seg[rows - padding:] = -1
    routing = _routing(rows, experts, top)
    X.route(z[:, :experts], seg, routing, scale, x, placed)
    return routing, zn[:, :experts]


@pytest.mark.parametrize("copies", [False, True])
@pytest.mark.parametrize("rows,experts,top,padding", [(1, 1, 1, 0), (3, 5, 2, 1), (9, 300, 9, 0), (700, 18, 4, 100), (33, 8, 8, 2), (16, 64, 1, 16)])
def test_route(rows, experts, top, padding, copies):
    rng = np.random.default_rng(rows)
    x, xn = _rand(rng, rows, 72)
    placed = torch.full((rows * top, 72), 9.0, device="cuda", dtype=torch.bfloat16) if copies else None
    routing, z = _route(rng, rows, experts, top, padding, x=x, placed=placed)
    real = rows - padding
    chosen, weight = O.route(z[:real], top, 2.5)
    assert np.array_equal(routing.chosen.cpu().numpy()[:real], chosen)
    _close(routing.weight[:real], weight, 1e-6) if real else None
    cu, token, place = (t.cpu().numpy() for t in (routing.cu, routing.token_of, routing.place_of))
    assert np.array_equal(np.diff(cu), np.bincount(chosen.ravel(), minlength=experts)) and cu[0] == 0
    assert (place[real:] == -1).all() and sorted(place[:real].ravel()) == list(range(real * top))
    for t in range(real):
        for k in range(top):
            e = chosen[t, k]
            assert cu[e] <= place[t, k] < cu[e + 1] and token[place[t, k]] == t
    assert int(routing.counters.abs().max()) == 0
    if copies:
        got = placed.double().cpu().numpy()
        assert np.array_equal(got[:real * top], xn[token[:real * top]]) and (got[real * top:] == 9.0).all()


def test_equal_logits_go_to_the_lower_index():
    from cacheir_b200 import expert_ops as X

    z = torch.tensor([[1.0, 3.0, 3.0, 1.0, 3.0], [0.0] * 5], device="cuda")
    routing = _routing(2, 5, 4)
    X.route(z, torch.zeros(2, device="cuda", dtype=torch.int32), routing, 1.0)
    assert routing.chosen.cpu().tolist() == [[1, 2, 4, 0], [0, 1, 2, 3]]


@pytest.mark.parametrize("rows,experts,top,n,k", [(1, 4, 2, 16, 8), (5, 3, 2, 136, 72), (40, 7, 3, 64, 264), (300, 5, 2, 256, 128), (600, 9, 4, 40, 64),
                                                  (900, 2, 2, 24, 512), (64, 40, 8, 520, 96), (17, 6, 6, 128, 1024), (65, 3, 1, 200, 136), (2300, 2, 2, 72, 64)])
def test_grouped_products(rows, experts, top, n, k):
    from cacheir_b200 import expert_ops as X
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(rows + n)
    x, xn = _rand(rng, rows, k)
    placed = torch.zeros((rows * top, k), device="cuda", dtype=torch.bfloat16)
    routing, _ = _route(rng, rows, experts, top, padding=rows // 5, x=x, placed=placed)
    cu, token = routing.cu.cpu().numpy(), routing.token_of.cpu().numpy()
    used = cu[-1]
    w, wn = _rand(rng, experts * n, k, scale=1.5 * k ** -0.5)
    expert = np.searchsorted(cu, np.arange(used), side="right") - 1

    def product(values):
        return np.stack([wn[e * n:(e + 1) * n] @ v for e, v in zip(expert, values)])
    y = product(xn[token[:used]])
    for source, by_row in [(placed, False)] + ([(x, True)] if rows <= X.grouped_all_rows() else []):
        out = torch.full((routing.places, n), 3.0, device="cuda", dtype=torch.bfloat16)
        X.grouped_gemm(source, w, out, routing, by_row=by_row)
        _close(out[:used], y, 5e-3)
        assert float((out[used:] - 3).abs().max() if used < routing.places else 0) == 0.0
        half = torch.empty((routing.places, n // 2), device="cuda", dtype=torch.bfloat16)
        X.grouped_gemm(source, w, half, routing, by_row=by_row, epilogue=H.DENSE_CLAMPED_GLU, limit=0.8)
        g, u = np.minimum(y[:, 0::2], 0.8), np.clip(y[:, 1::2], -0.8, 0.8)
        _close(half[:used], g * O.sigmoid(1.702 * g) * (u + 1), 6e-3)
        X.grouped_gemm(source, w, half, routing, by_row=by_row, epilogue=H.DENSE_SWIGLU)
        _close(half[:used], y[:, 0::2] * O.sigmoid(y[:, 0::2]) * y[:, 1::2], 6e-3)
    f32 = torch.empty((routing.places, n), device="cuda")
    X.grouped_simple(x.float(), w.float(), f32, routing, gather=True)
    _close(f32[:used], y, 3e-6)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("rows,width,top,shared", [(1, 8, 1, False), (7, 90, 3, True), (20, 1024, 4, True), (3, 12004, 2, True)])
def test_combine(rows, width, top, shared, dtype):
    from cacheir_b200 import expert_ops as X
    from cacheir_b200 import hybrid_ops as H

    td, tol = DTYPES[dtype]
    rng = np.random.default_rng(width)
    routing, z = _route(rng, rows, 6, top)
    chosen, weight = O.route(z, top, 2.5)
    y, yn = _rand(rng, rows * top, width, dtype=td)
    s, sn = _rand(rng, rows, width, dtype=td)
    res, rn = _rand(rng, rows, width, dtype=torch.float32)
    w, wn = _rand(rng, width, dtype=torch.float32)
    place = routing.place_of.cpu().numpy()
    m = np.einsum("tk,tkc->tc", weight, yn[place]) + (sn if shared else 0)
    want = rn + O.rms(m, 1e-3) * wn
    out = torch.empty((rows, width), device="cuda", dtype=td)
    X.combine_residual_rms(res, y, routing, s if shared else None, w, 1e-3, H.Next(out))
    _close(res, want, 5e-6)
    _close(out, want, 5e-3)


# ---- tied attention --------------------------------------------------------------------------------------------------------
def _attend(rng, shape, portions, *, dtype, kernel, size=None, keep=0, cap=24.0, scale=None, sink=True, gate=True, splits=0, base=1000.0,
            plant=None, eps=1e-5):
    """Sequences in shuffled pages: all but the last portion's tokens are cached first, then the portion runs through
    `kernel`. portions: (cached, new) per sequence. Returns (got, want) rows of the new tokens."""
    from cacheir_b200 import expert_ops as X
    from cacheir_b200.hybrid_ops import Rows
    from cacheir_b200.ragged import rotate_half_table

    heads, groups, dim, rot = shape
    td, _ = DTYPES[dtype]
    scale = 1.5 * dim ** -0.5 if scale is None else scale
    total = [a + b for a, b in portions]
    width = max((n + PAGE - 1) // PAGE for n in total) + 1
    slots = sum((n + PAGE - 1) // PAGE for n in total) + 3
    order = rng.permutation(slots)
    table = np.full((len(portions), width), -1, np.int32)
    at = 0
    for i, n in enumerate(total):
        pages = (n + PAGE - 1) // PAGE
        table[i, :pages] = order[at:at + pages]
        at += pages
    pool = torch.full((slots, groups, PAGE, dim + rot), float("nan"), device="cuda", dtype=td)      # (unwritten rows must not matter)
    inv = torch.full((slots, groups, PAGE), float("nan"), device="cuda")
    q, k, g, qn, kn, gn = [], [], [], [], [], []
    for n in total:
        a = rng.standard_normal((n, heads, dim)) * rng.uniform(0.5, 2.0)
        b = rng.standard_normal((n, groups, dim)) * rng.uniform(0.5, 2.0)
        if plant is not None:
            plant(a, b)
        for lst, ref, v in ((q, qn, a), (k, kn, b), (g, gn, rng.standard_normal((n, heads, dim)))):
            t = torch.from_numpy(v.astype(np.float32)).to(td)
            lst.append(t)
            ref.append(t.double().numpy())
    freq = O.frequencies(rot, base)
    sinks, sinkn = _rand(rng, heads, dtype=torch.float32)
    longest = max(total)
    rope = torch.from_numpy(rotate_half_table(longest, rot, base)).cuda() if rot else None

    def run(pick, name):
        """Rows of `pick` = (first, last + 1) per sequence."""
        rows = [(s, t) for s, (lo, hi) in enumerate(pick) for t in range(lo, hi)]
        if not rows:
            return None
        pad = 0 if name in ("step", "simple_step") else 3
        seg = torch.tensor([s for s, _ in rows] + [-1] * pad, device="cuda", dtype=torch.int32)
        pos = torch.tensor([t for _, t in rows] + [0] * pad, device="cuda", dtype=torch.int32)
        cu = torch.tensor(np.cumsum([0] + [hi - lo for lo, hi in pick]), device="cuda", dtype=torch.int32)
        meta = Rows(pos, seg, cu, torch.from_numpy(table).cuda(), torch.zeros(len(pick), device="cuda", dtype=torch.int32), name == "step")
        args = X.tied_args(meta, pool, inv, heads=heads, kv_heads=groups, dim=dim, rot_dims=rot, window=size or 1 << 30, keep_first=keep,
                           scale=scale, softcap=cap, sink=sinks if sink else None)
        cols = (heads * dim * 2 + groups * dim + 7) // 8 * 8
        x = torch.zeros((len(rows) + pad, cols), dtype=td)
        for i, (s, t) in enumerate(rows):
            x[i, :heads * dim] = q[s][t].flatten()
            x[i, heads * dim:(heads + groups) * dim] = k[s][t].flatten()
            x[i, (heads + groups) * dim:(2 * heads + groups) * dim] = g[s][t].flatten()
        x = x.cuda()
        qp = torch.full((len(rows) + pad, heads * X.query_width(dim, rot)), float("nan"), device="cuda", dtype=td)
        X.tied_prepare(args, x[:, :heads * dim], x[:, heads * dim:(heads + groups) * dim], qp, eps=eps, table=rope)
        out = torch.zeros((len(rows) + pad, heads * dim), device="cuda", dtype=td)
        gates = x[:, (heads + groups) * dim:(2 * heads + groups) * dim] if gate else None
        if name == "step":
            X.tied_attention_step(args, qp, gates, out, splits=splits)
        elif name == "prompt":
            X.tied_attention_prompt(args, qp, gates, out)
        elif name != "fill":
            X.tied_attention_simple(args, qp, gates, out)
        return out[:len(rows)]

    run([(0, a) for a, _ in portions], "fill")
    got = run([(a, n) for (a, _), n in zip(portions, total)], kernel).double().cpu().numpy()
    want = []
    for s, (a, _) in enumerate(portions):
        n = total[s]
        qq, kk = O.rms(O.rotate_half(qn[s], freq), eps), O.rms(O.rotate_half(kn[s], freq), eps)
        mask = O.seen(n, size, keep)
        o = np.empty((n, heads, dim))
        for h in range(heads):
            e = h // (heads // groups)
            p = O.sink_softmax(O.softcap((qq[:, h] @ kk[:, e].T) * scale, cap), mask, sinkn[h] if sink else None)
            o[:, h] = p @ kn[s][:, e]
        if gate:
            o = o * O.sigmoid(gn[s])
        want.append(o[a:].reshape(n - a, heads * dim))
    return got, np.concatenate(want)


def _agree(got, want, tol):
    assert np.isfinite(got).all()
    scale = np.sqrt((want ** 2).mean())
    err = np.sqrt(((got - want) ** 2).mean(axis=1)) / scale
    assert err.max() <= tol, (int(err.argmax()), float(err.max()))


SHAPES = [(6, 2, 64, 16), (8, 1, 128, 64), (3, 3, 32, 32), (6, 2, 40, 24), (20, 1, 128, 128), (2, 1, 256, 64), (4, 4, 192, 96), (1, 1, 8, 8), (34, 2, 72, 0),
          (160, 1, 16, 8)]
MASKS = [dict(size=37, keep=3), dict(size=None, keep=0), dict(size=1, keep=70), dict(size=200, keep=64), dict(size=64, keep=1, cap=None),
         dict(size=90, keep=5, cap=60.0, scale=1.0), dict(size=130, keep=0, cap=4.0, sink=False), dict(size=65, keep=2, gate=False)]
PORTIONS = [(0, 5), (70, 2), (0, 150), (129, 64), (63, 1), (200, 33), (64, 65)]


@pytest.mark.parametrize("mask", MASKS, ids=str)
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_attention_over_portions(shape, mask):
    rng = np.random.default_rng(shape[2])
    got, want = _attend(rng, shape, PORTIONS, dtype="bfloat16", kernel="prompt", **mask)
    _agree(got, want, 4e-2 if mask.get("scale") else 2e-2)      # (a score's rounding error grows with its scale)


@pytest.mark.parametrize("splits", [0, 1, 3])
@pytest.mark.parametrize("mask", MASKS, ids=str)
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_attention_of_single_tokens(shape, mask, splits):
    rng = np.random.default_rng(shape[2] + splits)
    portions = [(n, 1) for n in (0, 1, 63, 64, 127, 130, 300)]
    got, want = _attend(rng, shape, portions, dtype="bfloat16", kernel="step", splits=splits, **mask)
    _agree(got, want, 4e-2 if mask.get("scale") else 2e-2)      # (a score's rounding error grows with its scale)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("mask", MASKS[:6], ids=str)
@pytest.mark.parametrize("shape", [(6, 2, 64, 16), (3, 1, 10, 6), (2, 2, 7, 0), (1, 1, 1, 0), (5, 1, 72, 70)], ids=str)
def test_plain_attention(shape, mask, dtype):
    rng = np.random.default_rng(shape[0])
    got, want = _attend(rng, shape, [(0, 5), (70, 2), (0, 131)], dtype=dtype, kernel="simple", **mask)
    _agree(got, want, DTYPES[dtype][1] * (3 if mask.get("scale") else 1.5))


@pytest.mark.parametrize("kernel", ["prompt", "step", "simple"])
@pytest.mark.parametrize("where", ["window_in", "window_out", "first_in", "first_out", "page_edge"])
def test_one_key_that_stands_out(kernel, where):
    """A single key meets the last query with a score far above the rest, just inside or outside what it may see."""
    size, keep, n = 75, 6, 201
    key = {"window_in": n - size, "window_out": n - size - 1, "first_in": keep - 1, "first_out": keep, "page_edge": 128}[where]
    freq = O.frequencies(32, 1000.0)

    def plant(q, k):
        x = np.ones(64)                   # rotated back by the distance, so that key and query meet in phase at the end
        half = 16
        angle = (n - 1 - key) * freq
        u, v = x[:half], x[half:32]
        back = np.concatenate([u * np.cos(angle) - v * np.sin(angle), v * np.cos(angle) + u * np.sin(angle), x[32:]])
        q[n - 1] = x
        k[key] = back * 3.0
    rng = np.random.default_rng(3)
    got, want = _attend(rng, (2, 1, 64, 32), [(n - 1, 1)], dtype="float32" if kernel == "simple" else "bfloat16", kernel=kernel, size=size, keep=keep,
                        scale=0.2, cap=30.0, plant=plant, sink=False, gate=False, base=1000.0)
    lead = np.abs(want.reshape(-1, 64)).mean()
    assert (lead > 1.5) == (where in ("window_in", "first_in", "page_edge")), lead      # the oracle shows it
    _agree(got, want, 2e-2 if kernel != "simple" else 3e-5)


@pytest.mark.parametrize("value", [40.0, -40.0, 200.0])
def test_extreme_sinks(value, monkeypatch):
    """A sink far above every score empties the row, one far below changes nothing."""
    for kernel in ("prompt", "step"):
        def fixed(rng, *shape, scale=1.0, dtype=torch.bfloat16):
            t = torch.full(shape, value)
            return t.cuda(), t.double().numpy()
        monkeypatch.setattr(__import__(__name__), "_rand", fixed)
        got, want = _attend(np.random.default_rng(1), (6, 2, 64, 16), [(90, 1), (30, 1)], dtype="bfloat16", kernel=kernel, size=50, keep=2)
        assert np.isfinite(got).all()
        assert np.abs(got - want).max() <= 1.5e-2 * max(np.abs(want).max(), 1e-6) + 1e-12


def test_what_the_kernels_refuse():
    from cacheir_b200 import expert_ops as X
    from cacheir_b200._lib import CacheIRB200Error

    assert X.tied_prompt_supported(6, 2, 64, 16, 64, torch.bfloat16) and X.tied_step_supported(6, 2, 64, 16, 64, torch.bfloat16)
    for bad in ((6, 2, 60, 16), (6, 2, 64, 20), (4, 2, 264, 8), (4, 3, 64, 24)):
        assert not X.tied_prompt_supported(*bad, 64, torch.bfloat16) and not X.tied_step_supported(*bad, 64, torch.bfloat16)
    assert not X.tied_step_supported(6, 2, 64, 16, 16, torch.bfloat16) and not X.tied_prompt_supported(6, 2, 64, 16, 64, torch.float32)
    routing = _routing(2, 4, 2)
    with pytest.raises(CacheIRB200Error):
        X.grouped_gemm(torch.zeros((2, 12), device="cuda", dtype=torch.bfloat16), torch.zeros((32, 12), device="cuda", dtype=torch.bfloat16),
                       torch.zeros((4, 8), device="cuda", dtype=torch.bfloat16), routing, by_row=True)
    with pytest.raises(ValueError):
        X.route(torch.zeros((3, 4), device="cuda"), torch.zeros(3, device="cuda", dtype=torch.int32), routing, 1.0)
