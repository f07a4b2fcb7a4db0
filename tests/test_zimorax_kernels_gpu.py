"""What Zimorax adds to the kernels, one at a time against float64 statements of the same operator: talking-heads attention, short
convolutions, state spaces, the gated delta rule, layer norms, layer scale, squared ReLU."""
import numpy as np
import pytest
import torch

from oracle import zimorax as O

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


def _rows_close(got, want, tol):
    assert np.isfinite(got).all()
    err = np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean())
    assert err.max() <= tol, (int(err.argmax()), float(err.max()))


@pytest.fixture(autouse=True)
def _status():
    yield
    from cacheir_b200 import _lib
    assert _lib.group_device_status() == 0


def _pages(rng, lengths):
    """(page table with -1 where nothing is, slots): sequences in shuffled pages of a pool with some to spare."""
    counts = [(n + PAGE - 1) // PAGE for n in lengths]
    order = rng.permutation(sum(counts) + 3)
    table = np.full((len(lengths), max(counts) + 1), -1, np.int32)
    at = 0
    for i, n in enumerate(counts):
        table[i, :n] = order[at:at + n]
        at += n
    return table, sum(counts) + 3


def _meta(pick, table=None, slots=None, pad=0, decode=False):
    """Rows of `pick` = (first, last + 1) per sequence, with padding rows behind them."""
    from cacheir_b200.hybrid_ops import Rows

    rows = [(s, t) for s, (lo, hi) in enumerate(pick) for t in range(lo, hi)]
    seg = torch.tensor([s for s, _ in rows] + [-1] * pad, device="cuda", dtype=torch.int32)
    pos = torch.tensor([t for _, t in rows] + [0] * pad, device="cuda", dtype=torch.int32)
    cu = torch.tensor(np.cumsum([0] + [hi - lo for lo, hi in pick]), device="cuda", dtype=torch.int32)
    slots = torch.tensor([0] * len(pick) if slots is None else slots, device="cuda", dtype=torch.int32)
    table = np.zeros((len(pick), 1), np.int32) if table is None else table
    return rows, Rows(pos, seg, cu, torch.from_numpy(table).cuda(), slots, decode)


# ---- attention -------------------------------------------------------------------------------------------------------------
def _attend(rng, shape, portions, *, dtype, kernel, size=None, rot=0, yarn=None, scale=None, splits=0, plant=None):
    """All but the last portion's tokens are cached first, then the portion runs through `kernel`. shape: heads, key/value
    heads, key size, value size. Returns (got, want) of the new tokens."""
    from cacheir_b200 import mixer_ops as M
    from cacheir_b200.ragged import rotate_half_table, yarn_table

    heads, groups, dim, vdim = shape
    td, eps, base = DTYPES[dtype][0], 1e-5, 1000.0
    scale = 1.5 * dim ** -0.5 if scale is None else scale
    total = [a + b for a, b in portions]
    table, slots = _pages(rng, total)
    keys = torch.full((slots, PAGE, groups * dim), float("nan"), device="cuda", dtype=td)      # (unwritten rows must not matter)
    values = torch.full((slots, PAGE, groups * vdim), float("nan"), device="cuda", dtype=td)
    talkn = np.eye(heads) + rng.normal(0, 0.5 / np.sqrt(heads), (heads, heads))
    talk = torch.from_numpy(talkn.astype(np.float32)).to(torch.bfloat16).float()
    talkn, talk = talk.double().numpy(), talk.cuda()
    data, ref = [], []
    for n in total:
        parts = [rng.standard_normal((n, h * d)) for h, d in ((heads, dim), (groups, dim), (groups, vdim))]
        if plant is not None:
            plant(parts[0].reshape(n, heads, dim), parts[1].reshape(n, groups, dim))
        parts = [torch.from_numpy(p.astype(np.float32)).to(td) for p in parts]
        data.append(parts)
        ref.append([p.double().numpy() for p in parts])
    rope = None
    if rot:
        rope = rotate_half_table(max(total), rot, base) if yarn is None else yarn_table(max(total), rot, base, yarn)
        rope = torch.from_numpy(rope).cuda()
        freq, factor = O.yarn_frequencies(rot, base, None if yarn is None else dict(zip(("factor", "original", "fast", "slow"), yarn)))

    def run(pick, name):
        pad = 0 if name == "step" else 3
        rows, meta = _meta(pick, table, pad=pad, decode=name == "step")
        if not rows:
            return None
        args = M.talking_args(meta, keys, values, talk, heads=heads, kv_heads=groups, dim=dim, vdim=vdim, window=size or 1 << 30, scale=scale)
        sizes = [heads * dim, groups * dim, groups * vdim]
        x = torch.zeros((len(rows) + pad, (sum(sizes) + 7) // 8 * 8), dtype=td)
        for i, (s, t) in enumerate(rows):
            x[i, :sum(sizes)] = torch.cat([p[t] for p in data[s]])
        x = x.cuda()
        q, k, v = (x[:, sum(sizes[:i]):sum(sizes[:i + 1])] for i in range(3))
        mixed = name == "prompt"
        qp = torch.full((len(rows) + pad, heads * dim * (groups if mixed else 1)), float("nan"), device="cuda", dtype=td)
        M.talking_prepare(args, q, k, v, qp, eps=eps, table=rope, mixed=mixed)
        out = torch.zeros((len(rows) + pad, heads * vdim), device="cuda", dtype=td)
        if name == "step":
            M.talking_step(args, qp, out, splits=splits)
        elif name == "prompt":
            M.talking_prompt(args, qp, out)
        elif name == "simple":
            M.talking_simple(args, qp, out)
        return out[:len(rows)]

    run([(0, a) for a, _ in portions], "fill")
    got = run([(a, n) for (a, _), n in zip(portions, total)], kernel).double().cpu().numpy()
    want = []
    for (a, _), n, (q, k, v) in zip(portions, total, ref):
        q, k = (O.rotate_half(t.reshape(n, -1, dim), freq, factor) if rot else t.reshape(n, -1, dim) for t in (q, k))
        o = O.attend(q, k, O.rms(v.reshape(n, groups, vdim), eps), scale, talkn, O.seen(n, size))
        want.append(o[a:].reshape(n - a, heads * vdim))
    return got, np.concatenate(want)


# heads, key/value heads, key size, value size
SHAPES = [(6, 2, 40, 24), (3, 3, 16, 64), (2, 1, 128, 40), (4, 4, 64, 128), (2, 2, 256, 56), (4, 1, 72, 200), (1, 1, 8, 256), (20, 1, 64, 128), (5, 5, 24, 8),
          (16, 8, 128, 128), (34, 2, 16, 16), (9, 3, 56, 72), (8, 8, 8, 8)]
MASKS = [dict(size=37, rot=8, yarn=(8.0, 32.0, 4.0, 0.5)), dict(size=None), dict(size=1), dict(size=130, rot=8), dict(size=64, scale=0.05), dict(size=200, scale=-0.1)]
PORTIONS = [(0, 5), (70, 2), (0, 150), (129, 64), (63, 1), (200, 33), (64, 65)]


@pytest.mark.parametrize("mask", range(len(MASKS)))
@pytest.mark.parametrize("shape", SHAPES)
def test_prompt_attention(shape, mask):
    got, want = _attend(np.random.default_rng(1), shape, PORTIONS, dtype="bfloat16", kernel="prompt", **MASKS[mask])
    _rows_close(got, want, 2e-2)


@pytest.mark.parametrize("splits", [0, 1, 3, 8])
@pytest.mark.parametrize("shape", SHAPES)
def test_step_attention(shape, splits):
    for mask in MASKS[: 6 if splits == 0 else 2]:
        portions = [(n, 1) for n in (0, 1, 62, 63, 64, 65, 127, 300, 37)]
        got, want = _attend(np.random.default_rng(2), shape, portions, dtype="bfloat16", kernel="step", splits=splits, **mask)
        _rows_close(got, want, 2e-2)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", [(6, 2, 40, 24), (3, 1, 7, 5), (4, 4, 33, 12), (1, 1, 2, 1), (20, 5, 64, 64)])
def test_simple_attention(shape, dtype):
    for mask in (dict(size=37, rot=2, yarn=(3.0, 20.0, 2.0, 0.1)), dict(size=None), dict(size=1), dict(size=64, rot=2)):
        got, want = _attend(np.random.default_rng(3), shape, PORTIONS, dtype=dtype, kernel="simple", **mask)
        _rows_close(got, want, 2e-5 if dtype == "float32" else 2.5e-2)


@pytest.mark.parametrize("kernel", ["prompt", "step", "simple"])
@pytest.mark.parametrize("size,far", [(None, 0), (None, 63), (None, 64), (100, 99), (100, 100), (64, 63), (64, 64), (65, 64), (65, 65), (129, 128), (129, 129)])
def test_one_far_key_stands_out(kernel, size, far):
    """A key that one query meets with a large score, just inside or just outside the window, or far back. Only head 2 asks for it:
    the others hear of it through the mixture."""
    n, heads, groups, dim = 200, 4, 2, 64
    row = n - 1

    def plant(q, k):
        q *= 0.1
        k *= 0.1
        at = far if size is None else row - far
        q[row, 2] = 2.0
        k[at, 1] = 2.0
    portions = [(n - 1, 1)] if kernel == "step" else [(n - 40, 40)]
    got, want = _attend(np.random.default_rng(4), (heads, groups, dim, 32), portions, dtype="bfloat16", kernel=kernel, size=size, scale=0.05, plant=plant)
    _rows_close(got, want, 2e-2)
    other = None if size is None else size + (1 if far == size else -1)       # the test would notice a window that is one token off
    _, missed = _attend(np.random.default_rng(4), (heads, groups, dim, 32), portions, dtype="bfloat16", kernel=kernel, size=other, scale=0.05,
                        plant=plant if size is not None else None)
    assert np.abs(want[-1] - missed[-1]).max() > 0.1 * np.abs(want[-1]).max()


def test_rows_do_not_depend_on_their_neighbours():
    got, want = _attend(np.random.default_rng(5), (6, 2, 40, 24), [(100, 33)], dtype="bfloat16", kernel="prompt", size=50)
    cut, _ = _attend(np.random.default_rng(5), (6, 2, 40, 24), [(131, 2)], dtype="bfloat16", kernel="prompt", size=50)
    _rows_close(cut, got[-2:], 1e-2)
    _rows_close(got, want, 2e-2)


# ---- short convolution -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("channels,taps", [(40, 4), (7, 3), (640, 2), (12, 1), (9, 6), (516, 3), (1, 4), (16, 9)])
def test_short_convolution_in_portions(channels, taps, dtype):
    from cacheir_b200 import mixer_ops as M

    rng = np.random.default_rng(6)
    td, tol = DTYPES[dtype]
    lengths, cuts = (90, 1, 33, 70), ((0, 50, 52, 53, 90), (0, 1), (0, 2, 4, 33), (0, 64, 70))
    w, wn = _rand(rng, channels, taps, dtype=torch.float32)
    b, bn = _rand(rng, channels, dtype=torch.float32)
    xs = [_rand(rng, n, channels, dtype=td) for n in lengths]
    offset, slots = 8, [3, 0, 4, 1]
    size = (offset + (taps - 1) * channels + 3) // 4 * 4
    state = torch.full((5, size), float("nan"), device="cuda")          # (a new sequence does not read what a slot held before)
    stride = (channels + 11) // 4 * 4
    got = [[] for _ in lengths]
    for i in range(4):
        pick = [(c[i], c[i + 1]) if i + 1 < len(c) else (c[-1], c[-1]) for c in cuts]
        rows, meta = _meta(pick, slots=slots, pad=2)
        x = torch.zeros((len(rows) + 2, stride), device="cuda", dtype=td)[:, 4:4 + channels]
        for j, (s, t) in enumerate(rows):
            x[j] = xs[s][0][t]
        out = torch.zeros((len(rows) + 2, stride), device="cuda", dtype=td)[:, :channels]
        M.short_conv(meta, x, w, b if taps != 3 else None, state, offset, out)
        for j, (s, _) in enumerate(rows):
            got[s].append(out[j])
    for s, (_, xn) in enumerate(xs):
        _close(torch.stack(got[s]), O.causal_conv(xn, wn, bn if taps != 3 else None), tol)
    assert torch.isnan(state[2]).all() and torch.isnan(state[:, :offset]).all()


# ---- recurrences -----------------------------------------------------------------------------------------------------------
CUTS = [((0, 130), (0, 64, 65), (0, 1), (0, 300)), ((0, 2, 4, 70, 130), (0, 3, 65), (0, 1), (0, 129, 192, 193, 300)), ((0, 129, 130), (0, 64, 65), (0, 1), (0, 299, 300))]
LENGTHS, SLOTS = (130, 65, 1, 300), (2, 5, 0, 3)
STEP_LENGTHS = (40, 33, 40, 1)


def _recur(cuts, columns, run, decode):
    """Feeds the portions of every sequence step by step; `columns`: per sequence (host array [n, width], type) pairs. Returns the
    outputs per sequence."""
    got = [[] for _ in cuts]
    for i in range(max(len(c) for c in cuts) - 1):
        pick = [(s, (c[i], c[i + 1]) if i + 1 < len(c) else (c[-1], c[-1])) for s, c in enumerate(cuts)]
        if decode:                                    # only the live ones
            pick = [(s, p) for s, p in pick if p[0] < p[1]]
        pad = 0 if decode else 2
        rows, meta = _meta([p for _, p in pick], slots=[SLOTS[s] for s, _ in pick], pad=pad, decode=decode)
        rows = [(pick[s][0], t) for s, t in rows]
        x = [torch.zeros((len(rows) + pad, c.shape[1]), dtype=t) for c, t in columns[0]]
        for j, (s, t) in enumerate(rows):
            for dst, (src, _) in zip(x, columns[s]):
                dst[j] = torch.from_numpy(src[t])
        out = run(meta, [t.cuda() for t in x])
        for j, (s, _) in enumerate(rows):
            got[s].append(out[j])
    return [torch.stack(g) for g in got]


def _held(rng, td, *shape):
    """float32 array of values that `td` holds"""
    return torch.from_numpy(rng.standard_normal(shape).astype(np.float32)).to(td).float().numpy()


def _state_space(shape, kernel, dtype, cuts, rate=(-3.0, 1.0)):
    from cacheir_b200 import hybrid_ops as H

    heads, groups, dim, vdim = shape
    rng, td = np.random.default_rng(7), DTYPES[dtype][0]
    bias, biasn = _rand(rng, heads, dtype=torch.float32)
    skip, skipn = _rand(rng, heads, dtype=torch.float32)
    raten = rng.uniform(*rate, heads).astype(np.float32)
    rates = torch.from_numpy(raten).cuda()
    widths = (groups * dim, groups * dim, heads * vdim)
    lengths = [c[-1] for c in cuts]
    columns = [[(_held(rng, td, n, sum(widths)), td), (rng.normal(-1.0, 1.5, (n, heads)).astype(np.float32), torch.float32)] for n in lengths]
    state = torch.full((6, (heads * dim * vdim + 7) // 4 * 4), float("nan"), device="cuda")

    def run(meta, x):
        c, b, v = (x[0][:, sum(widths[:i]):sum(widths[:i + 1])] for i in range(3))
        out = torch.zeros((meta.rows, heads * vdim), device="cuda", dtype=td)
        steps = H.StepSizes(x[1], bias, rates)
        gates = [torch.empty((meta.rows, heads), device="cuda") for _ in range(2)]
        a = H.recurrence_args(meta, c, b, v, None, state, out, heads=heads, dim=dim, vdim=vdim, gated=(*gates, None), key_heads=groups, skip=skip, memory=False)
        if kernel == "step":
            H.state_space_step(a, steps)
            return out
        H.state_space_gates(a, steps, *gates)
        if kernel == "chunked":
            need = H.recurrence_workspace_bytes(meta.rows, meta.segments, heads, dim, vdim)
            H.recurrence_chunked(a, torch.full((need,), 255, device="cuda", dtype=torch.uint8) if need else None)
        else:
            H.recurrence_simple(a)
        return out
    for got, ((x, _), (z, _)), n in zip(_recur(cuts, columns, run, kernel == "step"), columns, lengths):
        c, b, v = np.split(x.astype(np.float64), np.cumsum(widths)[:2], axis=1)
        want = O.state_space(v.reshape(n, heads, vdim), b.reshape(n, groups, dim), c.reshape(n, groups, dim), O.softplus(z.astype(np.float64) + biasn),
                             raten.astype(np.float64), skipn)
        _close(got, want.reshape(n, -1), 2e-5 if dtype == "float32" else 1e-2)


PROMPT_KERNELS = [("chunked", "bfloat16"), ("simple", "bfloat16"), ("simple", "float32")]
PROMPT_SHAPES = [(6, 3, 48, 40), (4, 1, 64, 64), (2, 2, 16, 8), (4, 2, 128, 72), (3, 1, 112, 136)]
STEPS = [tuple(range(n + 1)) for n in STEP_LENGTHS]


@pytest.mark.parametrize("cuts", range(len(CUTS)))
@pytest.mark.parametrize("kernel,dtype", PROMPT_KERNELS)
@pytest.mark.parametrize("shape", PROMPT_SHAPES)
def test_state_space_prompts(shape, kernel, dtype, cuts):
    _state_space(shape, kernel, dtype, CUTS[cuts])


@pytest.mark.parametrize("rate", [(-9.0, -7.0), (3.0, 4.0)])
def test_state_space_with_long_and_short_memories(rate):
    _state_space((8, 4, 64, 32), "chunked", "bfloat16", CUTS[1], rate)
    _state_space((8, 4, 64, 32), "simple", "float32", CUTS[1], rate)


@pytest.mark.parametrize("shape", [(3, 3, 7, 5), (5, 1, 200, 33), (1, 1, 1, 1)])
def test_state_space_of_any_size(shape):
    _state_space(shape, "simple", "float32", CUTS[1])
    _state_space(shape, "simple", "bfloat16", CUTS[1])


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", [(6, 3, 48, 40), (4, 1, 64, 64), (2, 2, 16, 8), (4, 2, 7, 72), (1, 1, 300, 4), (1, 1, 3, 1024)])
def test_state_space_step(shape, dtype):
    _state_space(shape, "step", dtype, STEPS)


def _delta(shape, kernel, dtype, cuts, rate=(-3.0, 1.0), same=0.0):
    """`same`: how much all keys of a sequence have in common (they are far from orthogonal, and writes correct each other)."""
    from cacheir_b200 import mixer_ops as M

    heads, groups, dim, vdim = shape
    rng, td = np.random.default_rng(8), DTYPES[dtype][0]
    bias, biasn = _rand(rng, heads, dtype=torch.float32)
    raten = rng.uniform(*rate, heads).astype(np.float32)
    rates = torch.from_numpy(raten).cuda()
    norm, normn = _rand(rng, vdim, dtype=torch.float32)
    widths = (groups * dim, groups * dim, heads * vdim)
    lengths = [c[-1] for c in cuts]
    columns = []
    for n in lengths:
        x = rng.standard_normal((n, sum(widths)))
        x[:, widths[0]:2 * widths[0]] += same * rng.standard_normal(widths[0])
        x = torch.from_numpy(x.astype(np.float32)).to(td).float().numpy()
        columns.append([(x, td), (rng.normal(0, 1.5, (n, 2 * heads)).astype(np.float32), torch.float32), (_held(rng, td, n, heads * vdim), td)])
    state = torch.full((6, (heads * dim * vdim + 7) // 4 * 4), float("nan"), device="cuda")
    eps = 1e-5

    def run(meta, x):
        q, k, v = (x[0][:, sum(widths[:i]):sum(widths[:i + 1])] for i in range(3))
        out = torch.zeros((meta.rows, heads * vdim), device="cuda", dtype=td)
        a = M.delta_args(meta, q, k, v, x[1], bias, rates, state, out, heads=heads, key_heads=groups, dim=dim, vdim=vdim)
        if kernel == "step":
            M.delta_step(a, x[2], norm, eps)
        elif kernel == "chunked":
            M.delta_chunked(a, torch.full((M.delta_workspace_bytes(meta.rows, meta.segments, heads),), 255, device="cuda", dtype=torch.uint8))
        else:
            M.delta_simple(a)
        return out
    for got, ((x, _), (z, _), (g, _)), n in zip(_recur(cuts, columns, run, kernel == "step"), columns, lengths):
        q, k, v = np.split(x.astype(np.float64), np.cumsum(widths)[:2], axis=1)
        z, g = z.astype(np.float64), g.astype(np.float64)
        o = O.delta_rule(O.unit(q.reshape(n, groups, dim)) * dim ** -0.5, O.unit(k.reshape(n, groups, dim)), v.reshape(n, heads, vdim), O.sigmoid(z[:, :heads]),
                         np.exp(-np.exp(raten.astype(np.float64)) * O.softplus(z[:, heads:] + biasn)))
        if kernel == "step":
            o = O.rms(o, eps) * normn * O.silu(g).reshape(n, heads, vdim)
        _close(got, o.reshape(n, -1), 3e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("cuts", range(len(CUTS)))
@pytest.mark.parametrize("kernel,dtype", PROMPT_KERNELS)
@pytest.mark.parametrize("shape", PROMPT_SHAPES)
def test_delta_rule_prompts(shape, kernel, dtype, cuts):
    _delta(shape, kernel, dtype, CUTS[cuts])


@pytest.mark.parametrize("kernel,dtype", [("chunked", "bfloat16"), ("simple", "float32")])
@pytest.mark.parametrize("rate,same", [((-9.0, -7.0), 0.0), ((-9.0, -7.0), 3.0), ((2.0, 3.0), 1.0), ((-3.0, 0.0), 10.0)])
def test_delta_rule_with_long_memories_and_parallel_keys(kernel, dtype, rate, same):
    _delta((40, 8, 64, 32) if kernel == "chunked" else (4, 2, 64, 32), kernel, dtype, CUTS[1], rate, same)


@pytest.mark.parametrize("shape", [(3, 3, 7, 5), (5, 1, 200, 33), (1, 1, 1, 1)])
def test_delta_rule_of_any_size(shape):
    _delta(shape, "simple", "float32", CUTS[1])
    _delta(shape, "simple", "bfloat16", CUTS[1])


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", [(6, 3, 48, 40), (4, 1, 64, 64), (2, 2, 128, 128), (4, 2, 7, 72), (1, 1, 300, 4), (1, 1, 3, 1024), (2, 1, 256, 256)])
def test_delta_step(shape, dtype):
    _delta(shape, "step", dtype, STEPS, same=1.0)


# ---- rows ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("width", [16, 90, 136, 1028, 4096, 9000])
def test_scaled_residual_and_layer_norms(width, dtype):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(9)
    td, tol = DTYPES[dtype]
    rows, eps = 5, 1e-4
    y, yn = _rand(rng, rows, width, dtype=td)
    w, wn = _rand(rng, width, dtype=torch.float32)
    s, sn = _rand(rng, width, dtype=torch.float32)
    for scale, norm in ((s, H.LayerNorm(w, eps)), (None, H.LayerNorm(w, eps)), (s, H.RmsNorm(w, eps)), (s, None), (s, "none")):
        x = _rand(rng, rows, width, dtype=torch.float32)[0] + 3.0                 # (a mean to take off)
        xn = x.double().cpu().numpy()
        out = torch.zeros((rows, width), device="cuda", dtype=td)
        H.residual_add(x, y, None if norm == "none" else H.Next(out, norm), scale)
        want = xn + yn * (1.0 if scale is None else sn)
        _close(x, want, 1e-6)
        if norm != "none":
            want = want if norm is None else O.layer_norm(want, wn, eps) if isinstance(norm, H.LayerNorm) else O.rms(want, eps) * wn
            _close(out, want, tol)
    index = torch.tensor([4, 0, 4], device="cuda", dtype=torch.int32)
    out = torch.zeros((3, width), device="cuda", dtype=td)
    H.layer_norm_rows(x, w, eps, out, index)
    _close(out, O.layer_norm(x.double().cpu().numpy()[[4, 0, 4]], wn, eps), tol)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_layer_norm_behind_a_pair_of_norms(dtype):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(13)
    td, tol = DTYPES[dtype]
    (x, xn), (w, wn) = _rand(rng, 4, 96, dtype=torch.float32), _rand(rng, 96, dtype=torch.float32)
    (a, an), (b, bn) = _rand(rng, 4, 96, dtype=td), _rand(rng, 4, 96, dtype=td)
    out = torch.zeros((4, 96), device="cuda", dtype=td)
    H.residual_rms_pair(x, a, w, b, w, 0.5, 1e-5, H.Next(out, H.LayerNorm(w, 1e-5)))
    _close(out, O.layer_norm(xn + 0.5 * wn * (O.rms(an, 1e-5) + O.rms(bn, 1e-5)), wn, 1e-5), tol)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("width", [16, 90, 1028])
def test_embedding_joins_the_stream(width, dtype):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(10)
    td = DTYPES[dtype][0]
    table, tn = _rand(rng, 11, width, dtype=td)
    ids = torch.tensor([3, 0, 10, 7], device="cuda")
    w, wn = _rand(rng, width, dtype=torch.float32)
    x, out = torch.zeros((4, width), device="cuda"), torch.zeros((4, width), device="cuda", dtype=td)
    H.scaled_embedding(table, ids, x, 1.0, H.Next(out, H.LayerNorm(w, 1e-5)))
    assert np.array_equal(x.double().cpu().numpy(), tn[[3, 0, 10, 7]])
    _close(out, O.layer_norm(tn[[3, 0, 10, 7]], wn, 1e-5), DTYPES[dtype][1])
    x, _ = _rand(rng, 4, width, dtype=torch.float32)
    joined = torch.zeros((4, 2 * width), device="cuda", dtype=td)
    H.join_embedding(x, table, ids, joined)
    assert np.array_equal(joined.double().cpu().numpy(), np.concatenate([x.to(td).double().cpu().numpy(), tn[[3, 0, 10, 7]]], axis=1))


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("cols,parts", [(240, 6), (72, 1), (4096, 8), (10, 5), (3000, 2), (700, 1), (33, 3), (2048, 16), (9000, 3)])
def test_gated_norms_in_parts(cols, parts, dtype):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(11)
    td, tol = DTYPES[dtype]
    rows, eps, size = 5, 1e-3, cols // parts
    o, on = _rand(rng, rows, cols, dtype=td)
    wide, gn = _rand(rng, rows, cols + 4, dtype=td)
    gate, gn = wide[:, 4:], gn[:, 4:]
    for shared in (False, True):
        for first in (False, True):
            w, wn = _rand(rng, size if shared else cols, dtype=torch.float32)
            out = torch.zeros((rows, cols), device="cuda", dtype=td)
            H.gated_parts_rms(o, gate, w, eps, out, parts=parts, gate_first=first)
            x = on * O.silu(gn) if first else on
            want = O.rms(x.reshape(rows, parts, size), eps).reshape(rows, cols) * (np.tile(wn, parts) if shared else wn)
            _close(out, want if first else want * O.silu(gn), tol)


@pytest.mark.parametrize("rows,n,k", [(3, 40, 24), (1, 1, 8), (70, 300, 136), (300, 264, 64)])
def test_squared_relu_product(rows, n, k):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(12)
    x, xn = _rand(rng, rows, k)
    w, wn = _rand(rng, n, k, scale=k ** -0.5)
    b, bn = _rand(rng, n, dtype=torch.float32)
    want = np.maximum(xn @ wn.T + bn, 0.0) ** 2
    out = torch.zeros((rows, (n + 7) // 8 * 8), device="cuda", dtype=torch.bfloat16)[:, :n]
    H.dense_gemm(x, w, out, epilogue=H.DENSE_RELU2, bias=b)
    _close(out, want, 1e-2)
    for td, tol in DTYPES.values():
        y = torch.zeros((rows, n), device="cuda", dtype=td)
        H.dense_simple(x.to(td), w.to(td), y, bias=b)
        H.relu2_cols(y, n)
        _close(y, want, tol)
