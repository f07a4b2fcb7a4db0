"""What Rekodra adds to the kernels, one at a time against float64 statements of the same operator: rows with keys and values
of their own, weighted norms, matrix memory, softmax routing, residual rows."""
import numpy as np
import pytest
import torch

from oracle import rekodra as O

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


def _meta(pick, table, slots=None, pad=0, decode=False):
    """Rows of `pick` = (first, last + 1) per sequence, with padding rows behind them."""
    from cacheir_b200.hybrid_ops import Rows

    rows = [(s, t) for s, (lo, hi) in enumerate(pick) for t in range(lo, hi)]
    seg = torch.tensor([s for s, _ in rows] + [-1] * pad, device="cuda", dtype=torch.int32)
    pos = torch.tensor([t for _, t in rows] + [0] * pad, device="cuda", dtype=torch.int32)
    cu = torch.tensor(np.cumsum([0] + [hi - lo for lo, hi in pick]), device="cuda", dtype=torch.int32)
    slots = torch.tensor([0] * len(pick) if slots is None else slots, device="cuda", dtype=torch.int32)
    return rows, Rows(pos, seg, cu, torch.from_numpy(table).cuda(), slots, decode)


# ---- attention -------------------------------------------------------------------------------------------------------------
def _attend(rng, shape, portions, *, dtype, kernel, own, whole, size=None, rot=0, scale=None, sink=True, splits=0, spread=0.3, plant=None,
            bounded=True):
    """All but the last portion's tokens are cached first, then the portion runs through `kernel`. shape: heads, key/value
    heads, key size, value size; `own`: values of their own, else they are the keys. Returns (got, want) of the new tokens."""
    from cacheir_b200 import expert_ops as X
    from cacheir_b200.ragged import rotate_half_table

    heads, groups, dim, vdim = shape
    td, eps, base = DTYPES[dtype][0], 1e-5, 1000.0
    scale = 1.5 * dim ** -0.5 if scale is None else scale
    total = [a + b for a, b in portions]
    table, slots = _pages(rng, total)
    key_dim = dim if own else None
    width = X.row_layout(vdim, rot, key_dim)[0]
    pool = torch.full((slots, groups, PAGE, width), float("nan"), device="cuda", dtype=td)      # (unwritten rows must not matter)
    inv = torch.full((slots, groups, PAGE), float("nan"), device="cuda")
    qw, qwn = (torch.from_numpy((1 + spread * rng.standard_normal(heads * dim if whole else dim)).astype(np.float32)) for _ in range(2))
    kw = torch.from_numpy((1 + spread * rng.standard_normal(groups * dim if whole else dim)).astype(np.float32))
    qwn, kwn = qw.double().numpy(), kw.double().numpy()
    qw, kw = qw.cuda(), kw.cuda()
    data, ref = [], []
    for n in total:
        parts = [rng.standard_normal((n, h * d)) * rng.uniform(0.5, 2.0) for h, d in ((heads, dim), (groups, dim), (groups, vdim))]
        if plant is not None:
            plant(parts[0].reshape(n, heads, dim), parts[1].reshape(n, groups, dim), qwn, kwn)
        parts = [torch.from_numpy(p.astype(np.float32)).to(td) for p in parts]
        data.append(parts)
        ref.append([p.double().numpy() for p in parts])
    sinks, sinkn = _rand(rng, heads, dtype=torch.float32)
    rope = torch.from_numpy(rotate_half_table(max(total), rot, base)).cuda() if rot else None
    largest = float(np.abs(qwn).max() * np.abs(kwn).max()) * dim * ((heads * groups) ** 0.5 if whole else 1.0)

    def run(pick, name):
        pad = 0 if name == "step" else 3
        rows, meta = _meta(pick, table, pad=pad, decode=name == "step")
        if not rows:
            return None
        args = X.tied_args(meta, pool, inv, heads=heads, kv_heads=groups, dim=vdim, rot_dims=rot, window=size or 1 << 30, keep_first=0, scale=scale,
                           softcap=None, sink=sinks if sink else None, key_dim=key_dim, reach=largest if bounded else 0.0)
        sizes = [heads * dim, groups * dim, groups * vdim if own else 0]
        x = torch.zeros((len(rows) + pad, (sum(sizes) + 7) // 8 * 8), dtype=td)
        for i, (s, t) in enumerate(rows):
            x[i, :sum(sizes)] = torch.cat([p[t] for p in data[s][:3 if own else 2]])
        x = x.cuda()
        q, k, v = (x[:, sum(sizes[:i]):sum(sizes[:i + 1])] for i in range(3))
        qp = torch.full((len(rows) + pad, heads * X.query_width(vdim, rot, key_dim)), float("nan"), device="cuda", dtype=td)
        X.tied_prepare(args, q, k, qp, eps=eps, table=rope, v=v if own else None, q_weight=qw, k_weight=kw, whole=whole)
        out = torch.zeros((len(rows) + pad, heads * vdim), device="cuda", dtype=td)
        if name == "step":
            X.tied_attention_step(args, qp, None, out, splits=splits)
        elif name == "prompt":
            X.tied_attention_prompt(args, qp, None, out)
        elif name == "simple":
            X.tied_attention_simple(args, qp, None, out)
        return out[:len(rows)]

    run([(0, a) for a, _ in portions], "fill")
    got = run([(a, n) for (a, _), n in zip(portions, total)], kernel).double().cpu().numpy()
    want = []
    for (a, _), n, (q, k, v) in zip(portions, total, ref):
        if whole:
            qn, kn = (O.rms(q, eps) * qwn).reshape(n, heads, dim), (O.rms(k, eps) * kwn).reshape(n, groups, dim)
        else:
            qn, kn = O.rms(q.reshape(n, heads, dim), eps) * qwn, O.rms(k.reshape(n, groups, dim), eps) * kwn
        qn, kn = O.rotate_half(qn, rot, base), O.rotate_half(kn, rot, base)
        o = O.attend(qn, kn, (v if own else k).reshape(n, groups, vdim), scale, O.seen(n, size), sinkn if sink else None)
        want.append(o[a:].reshape(n - a, heads * vdim))
    return got, np.concatenate(want)


# heads, key/value heads, key size, value size
OWN = [(6, 2, 40, 24), (3, 3, 16, 64), (2, 1, 128, 40), (4, 4, 64, 128), (2, 2, 256, 56), (4, 1, 72, 200), (1, 1, 8, 256), (20, 1, 256, 256), (5, 5, 24, 8)]
TIED = [(6, 2, 64), (8, 1, 128), (20, 4, 40), (2, 1, 256), (40, 2, 72)]
OWN_MASKS = [dict(size=37, sink=False), dict(size=None), dict(size=1, sink=False), dict(size=130, sink=False, rot=8, bounded=False), dict(size=64, scale=0.05)]
PORTIONS = [(0, 5), (70, 2), (0, 150), (129, 64), (63, 1), (200, 33), (64, 65)]
STEPS = [(n, 1) for n in (0, 1, 63, 64, 127, 130, 300)]


@pytest.mark.parametrize("kernel,portions", [("prompt", PORTIONS), ("step", STEPS)])
@pytest.mark.parametrize("mask", OWN_MASKS, ids=str)
@pytest.mark.parametrize("shape", OWN, ids=str)
def test_attention_with_values_of_their_own(shape, mask, kernel, portions):
    from cacheir_b200 import expert_ops as X
    rng = np.random.default_rng(shape[2] + shape[3])
    if kernel == "prompt":
        assert X.tied_prompt_supported(shape[0], shape[1], shape[3], 0, PAGE, torch.bfloat16, shape[2])
    for whole in (False, True):
        got, want = _attend(rng, shape, portions, dtype="bfloat16", kernel=kernel, own=True, whole=whole, **mask)
        _rows_close(got, want, 2e-2)


@pytest.mark.parametrize("kernel,portions", [("prompt", PORTIONS), ("step", STEPS)])
@pytest.mark.parametrize("rot", [0, 16, 40])
@pytest.mark.parametrize("shape", TIED, ids=str)
def test_attention_with_one_norm_over_all_heads(shape, rot, kernel, portions):
    rng = np.random.default_rng(shape[2] + rot)
    got, want = _attend(rng, shape + shape[2:], portions, dtype="bfloat16", kernel=kernel, own=False, whole=True, rot=rot)
    _rows_close(got, want, 2e-2)


@pytest.mark.parametrize("splits", [1, 2, 5])
def test_splits_of_rows_with_values_of_their_own(splits):
    rng = np.random.default_rng(splits)
    got, want = _attend(rng, (4, 2, 56, 88), STEPS, dtype="bfloat16", kernel="step", own=True, whole=False, splits=splits)
    _rows_close(got, want, 2e-2)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("own,whole", [(True, False), (True, True), (False, True), (False, False)])
@pytest.mark.parametrize("shape", [(6, 2, 40, 24), (3, 1, 10, 7), (2, 2, 7, 20), (1, 1, 2, 1)], ids=str)
def test_plain_attention(shape, own, whole, dtype):
    rng = np.random.default_rng(shape[0])
    shape = shape if own else shape[:3] + shape[2:3]
    for size, rot in ((None, shape[2] // 4 * 2), (13, 0)):
        got, want = _attend(rng, shape, [(0, 5), (70, 2), (0, 131)], dtype=dtype, kernel="simple", own=own, whole=whole, size=size, rot=rot)
        _rows_close(got, want, DTYPES[dtype][1] * 1.5)


@pytest.mark.parametrize("kernel", ["prompt", "step", "simple"])
@pytest.mark.parametrize("where", ["inside", "outside", "page_first", "page_last", "far"])
def test_one_key_that_stands_out(kernel, where):
    """A single key meets the last query with a score far above the rest: just inside or outside the window, at a page's
    edges, or hundreds of keys away without one."""
    size, n = (None if where == "far" else 75), 401
    key = {"inside": n - 75, "outside": n - 76, "page_first": 384, "page_last": 383, "far": 3}[where]

    def plant(q, k, qw, kw):
        q[n - 1] = 3.0 * np.sign(qw)
        k[key] = 3.0 * np.sign(kw)
    rng = np.random.default_rng(3)
    got, want = _attend(rng, (4, 2, 32, 40), [(n - 1, 1)], dtype="bfloat16", kernel=kernel, own=True, whole=False, size=size, scale=0.5,
                        sink=False, spread=0.05, plant=plant)
    _rows_close(got, want, 2e-2)
    plain, _ = _attend(np.random.default_rng(3), (4, 2, 32, 40), [(n - 1, 1)], dtype="bfloat16", kernel=kernel, own=True, whole=False, size=size,
                       scale=0.5, sink=False, spread=0.05)
    moved = np.abs(got - plain).max() > 0.5
    assert moved or where == "outside"


@pytest.mark.parametrize("kernel", ["prompt", "step"])
def test_references_that_move_far(kernel):
    """Scores without a known bound that grow by hundreds along the sequence, with and without a sink above them all."""
    def plant(q, k, qw, kw):
        k *= np.linspace(0.05, 1.0, len(k))[:, None, None] ** 2
        q += 4.0
        k += np.linspace(-2, 2, len(k))[:, None, None]
    for own, sink in ((True, True), (True, False), (False, True)):
        shape = (4, 2, 64, 64)
        portions = [(0, 300)] if kernel == "prompt" else [(299, 1), (130, 1)]
        got, want = _attend(np.random.default_rng(5), shape, portions, dtype="bfloat16", kernel=kernel, own=own, whole=True, scale=2.0, sink=sink,
                            spread=0.1, plant=plant, bounded=False)
        _rows_close(got, want, 0.12)           # (scores of hundreds: a key's rounding moves them by whole units)


# ---- matrix memory ---------------------------------------------------------------------------------------------------------
class Memory:
    """Random inputs of several sequences, run in portions through the kernels and as a whole through the oracle."""

    def __init__(self, heads, dim, vdim, lengths, *, dtype, seed, in_bias=(0.0, 1.5), forget=(0.0, 6.0), cap=8.0):
        rng = np.random.default_rng(seed)
        self.heads, self.dim, self.vdim, self.cap, self.eps = heads, dim, vdim, cap, 1e-4
        self.td = DTYPES[dtype][0]
        self.lengths, self.inputs, self.want = lengths, [], []
        f32 = torch.float32
        self.in_bias, ibn = _rand(rng, heads, scale=in_bias[1], dtype=f32)
        self.in_bias += in_bias[0]
        ibn = ibn + in_bias[0]
        self.forget_bias = torch.from_numpy(rng.uniform(*forget, heads).astype(np.float32)).cuda()
        self.norm, normn = _rand(rng, heads * vdim, dtype=f32)
        for n in lengths:
            q, k, v, g = (_rand(rng, n, heads * d, dtype=self.td) for d in (dim, dim, vdim, vdim))
            z, zn = _rand(rng, n, 2 * heads, scale=2.0, dtype=f32)
            self.inputs.append((q[0], k[0], v[0], g[0], z))
            gi = cap * np.tanh((zn[:, :heads] + ibn) / cap)
            gf = O.log_sigmoid(cap * np.tanh((zn[:, heads:] + self.forget_bias.double().cpu().numpy()) / cap))
            o = O.matrix_memory(q[1].reshape(n, heads, dim) * dim ** -0.5, k[1].reshape(n, heads, dim), v[1].reshape(n, heads, vdim), gi, gf)
            self.want.append((O.rms(o, self.eps).reshape(n, heads * vdim) * normn * O.sigmoid(g[1])))
        from cacheir_b200 import hybrid_ops as H
        self.H = H
        self.slots = [int(s) for s in rng.permutation(len(lengths) + 2)[:len(lengths)]]
        self.state = torch.full((len(lengths) + 2, H.memory_state_size(heads, dim, vdim)), 7.0, device="cuda")      # (what earlier owners left)

    def run(self, pick, form):
        """Tokens `pick` = (first, last + 1) per sequence; returns [rows, heads*vdim]."""
        H, heads, dim, vdim = self.H, self.heads, self.dim, self.vdim
        pad = 0 if form == "step" else 2
        rows, meta = _meta(pick, np.zeros((len(pick), 1), np.int32), self.slots, pad=pad, decode=form == "step")
        gathered = [torch.cat([x[i][lo:hi] for x, (lo, hi) in zip(self.inputs, pick)] + [self.inputs[0][i][:1]] * pad) for i in range(5)]
        x = torch.cat([t.to(self.td) for t in gathered[:4]] + [torch.zeros(len(rows) + pad, -sum(t.shape[1] for t in gathered[:4]) % 8, device="cuda", dtype=self.td)], 1)
        q, k, v, g = x[:, :sum(t.shape[1] for t in gathered[:4])].split([t.shape[1] for t in gathered[:4]], dim=1)
        gates = H.MemoryGates(gathered[4], self.in_bias, self.forget_bias, self.cap)
        out = torch.zeros((len(rows) + pad, heads * vdim), device="cuda", dtype=self.td)
        if form == "step":
            args = H.recurrence_args(meta, q, k, v, None, self.state, out, heads=heads, dim=dim, vdim=vdim, q_scale=dim ** -0.5)
            H.memory_step(args, gates, g, self.norm, self.eps)
            return out
        decay, take, maximum, normaliser = (torch.zeros((len(rows) + pad, heads), device="cuda") for _ in range(4))
        o = torch.zeros_like(out)
        args = H.recurrence_args(meta, q, k, v, None, self.state, o, heads=heads, dim=dim, vdim=vdim, gated=(decay, take, normaliser), q_scale=dim ** -0.5)
        H.memory_gates(args, gates, decay, take, maximum)
        if form == "chunked":
            need = H.recurrence_workspace_bytes(meta.rows, meta.segments, heads, dim, vdim)
            H.recurrence_chunked(args, torch.full((need,), 255, device="cuda", dtype=torch.uint8) if need else None)      # (NaNs)
        else:
            H.recurrence_simple(args)
        H.memory_norm(o, normaliser, maximum, g, self.norm, self.eps, out, heads=heads, vdim=vdim)
        return out[:len(rows)]

    def check(self, plan, tol):
        """plan: (form, tokens per sequence) one after the other."""
        at = [0] * len(self.lengths)
        for form, counts in plan:
            pick = [(a, min(a + c, n)) for a, c, n in zip(at, counts, self.lengths)]
            got = self.run(pick, form).double().cpu().numpy()
            _rows_close(got, np.concatenate([w[lo:hi] for w, (lo, hi) in zip(self.want, pick)]), tol)
            at = [hi for _, hi in pick]
        assert at == list(self.lengths)


MEMORY_SHAPES = [(3, 48, 40), (2, 128, 64), (1, 16, 200), (4, 64, 8), (2, 112, 136)]


@pytest.mark.parametrize("shape", MEMORY_SHAPES, ids=str)
def test_memory_prompts_on_the_tensor_cores(shape):
    m = Memory(*shape, (700, 64, 1, 65, 300, 256, 257), dtype="bfloat16", seed=shape[1])
    m.check([("chunked", (700,) * 7)], 1.5e-2)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", MEMORY_SHAPES[:2] + [(1, 1, 1), (5, 12, 18), (2, 20, 7), (1, 300, 33)], ids=str)
def test_memory_token_by_token_kernel(shape, dtype):
    m = Memory(*shape, (70, 1, 33), dtype=dtype, seed=shape[1])
    m.check([("simple", (70,) * 3)], 1e-4 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", [(3, 48, 40), (2, 128, 64), (2, 17, 4), (1, 300, 1024), (1, 1, 12)], ids=str)
def test_memory_portions_and_decoding_carry_the_state(shape, dtype):
    chunked = dtype == "bfloat16" and shape[1] % 16 == 0 and shape[1] <= 128
    form = "chunked" if chunked else "simple"
    m = Memory(*shape, (340, 10, 129), dtype=dtype, seed=shape[2])
    steps = [("step", (1, 1, 1))] * 4
    m.check([(form, (2, 3, 64))] + steps + [(form, (270, 0, 2)), (form, (57, 2, 57))] + steps[:1] + [("simple", (2, 0, 0))]
            + [(form, (340, 340, 340))], 1e-4 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("form", ["chunked", "simple", "step"])
def test_memory_starts_from_a_maximum_of_zero(form):
    """Input gates far below zero: the sums stay small beside exp(-m) = 1, so outputs are far below one over the normaliser;
    the first token shows it most."""
    m = Memory(2, 32, 32, (5, 1, 3) if form != "step" else (1, 1, 1), dtype="bfloat16", seed=2, in_bias=(-7.0, 0.3))
    m.eps = 1e-4
    m.check([(form, (5, 5, 5))], 1.5e-2)


@pytest.mark.parametrize("form", ["chunked", "simple"])
def test_memory_remembers_and_forgets(form):
    """Forget gates near one: the first token still counts after 900; near zero: only the last few do."""
    for forget in ((9.0, 12.0), (-6.0, -3.0)):
        m = Memory(2, 64, 32, (900, 300), dtype="bfloat16", seed=4, forget=forget, cap=15.0)
        m.check([(form, (520, 256)), (form, (900, 900))], 1.5e-2)


# ---- routing ---------------------------------------------------------------------------------------------------------------
def _routing(rows, experts, top):
    from cacheir_b200 import expert_ops as X

    def ints(*shape):
        return torch.full(shape, -7, device="cuda", dtype=torch.int32)
    return X.Routing(experts, top, torch.zeros(experts + 1, device="cuda", dtype=torch.int32), ints(experts + 1), ints(rows * top), ints(rows, top),
                     ints(rows, top), torch.empty((rows, top), device="cuda"))


def _route(rng, rows, experts, identity, top, groups, keep, padding=0, x=None, placed=None):
    from cacheir_b200 import expert_ops as X

    scored = experts + identity
    z, zn = _rand(rng, rows, scored + 1, dtype=torch.float32)
    c, cn = _rand(rng, scored, scale=0.3, dtype=torch.float32)
    seg = torch.arange(rows, device="cuda", dtype=torch.int32)
    if padding:
        seg[rows - padding:] = -1
    routing = _routing(rows, experts, top)
    X.route(z, seg, routing, 1.0, x, placed, X.SoftmaxRule(c, groups, keep, identity))
    return routing, O.route(zn[:, :scored], cn, top, groups, keep)


@pytest.mark.parametrize("copies", [False, True])
@pytest.mark.parametrize("rows,experts,identity,top,groups,keep,padding", [
    (1, 1, 0, 1, 1, 1, 0), (9, 5, 1, 2, 3, 2, 1), (40, 12, 4, 3, 2, 1, 0), (700, 30, 2, 4, 8, 3, 100), (33, 8, 0, 8, 4, 4, 2), (16, 240, 60, 9, 30, 5, 0),
    (16, 3, 3, 4, 6, 6, 16), (70, 2, 6, 3, 2, 2, 3)])
def test_softmax_routing(rows, experts, identity, top, groups, keep, padding, copies):
    from cacheir_b200 import expert_ops as X  # noqa: F401
    rng = np.random.default_rng(rows + experts)
    x, xn = _rand(rng, rows, 72)
    placed = torch.full((rows * top, 72), 9.0, device="cuda", dtype=torch.bfloat16) if copies else None
    routing, (chosen, weight) = _route(rng, rows, experts, identity, top, groups, keep, padding, x, placed)
    real = rows - padding
    chosen, weight = chosen[:real], weight[:real]
    assert np.array_equal(routing.chosen.cpu().numpy()[:real], chosen)
    if real:
        _close(routing.weight[:real], weight, 1e-6)
    cu, token, place = (t.cpu().numpy() for t in (routing.cu, routing.token_of, routing.place_of))
    tensors = chosen[chosen < experts]
    assert np.array_equal(np.diff(cu), np.bincount(tensors, minlength=experts)) and cu[0] == 0
    assert (place[real:] == -1).all() and (place[:real][chosen >= experts] == -2).all()
    assert sorted(place[:real][chosen < experts]) == list(range(len(tensors)))
    for t in range(real):
        for k in range(top):
            e = chosen[t, k]
            assert e >= experts or (cu[e] <= place[t, k] < cu[e + 1] and token[place[t, k]] == t)
    assert int(routing.counters.abs().max()) == 0
    if copies:
        got = placed.double().cpu().numpy()
        assert np.array_equal(got[:len(tensors)], xn[token[:len(tensors)]]) and (got[len(tensors):] == 9.0).all()


def test_dropped_groups_lose_even_to_negative_scores():
    from cacheir_b200 import expert_ops as X

    z = torch.tensor([[3.0, 0.0, 2.9, 2.8]], device="cuda")
    c = torch.tensor([0.0, -4.0, 0.0, 0.0], device="cuda")
    routing = _routing(1, 4, 2)
    X.route(z, torch.zeros(1, device="cuda", dtype=torch.int32), routing, 1.0, rule=X.SoftmaxRule(c, 2, 1, 0))
    assert routing.chosen.cpu().tolist() == [[0, 1]]
    _close(routing.weight, O.softmax(z.double().cpu().numpy())[:, :2], 1e-6)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("rows,width,top,shared,gated", [(1, 8, 1, False, False), (7, 90, 3, True, True), (20, 1024, 4, True, False), (3, 12004, 2, True, True)])
def test_combine_with_identity_experts_and_a_gated_shared_one(rows, width, top, shared, gated, dtype):
    from cacheir_b200 import expert_ops as X
    from cacheir_b200 import hybrid_ops as H

    td, _ = DTYPES[dtype]
    rng = np.random.default_rng(width)
    routing, (chosen, weight) = _route(rng, rows, 4, 4, top, 2, 2)
    y, yn = _rand(rng, rows * top, width, dtype=td)
    s, sn = _rand(rng, rows, width, dtype=td)
    x, xn = _rand(rng, rows, width, dtype=td)
    g, gn = _rand(rng, rows, 3, dtype=torch.float32)
    w, wn = _rand(rng, width, dtype=torch.float32)
    res, rn = _rand(rng, rows, width, dtype=torch.float32)
    place = routing.place_of.cpu().numpy()
    rows_of = np.where((chosen < 4)[..., None], yn[np.maximum(place, 0)], xn[:, None])
    want = rn + np.einsum("tk,tkc->tc", weight, rows_of) + (sn * (O.sigmoid(gn[:, 2:]) if gated else 1) if shared else 0)
    out = x                                       # (the next input may replace the one that identity experts return)
    X.combine_residual(res, y, routing, x, s if shared else None, g[:, 2] if gated else None, H.Next(out, H.RmsNorm(w, 1e-3)))
    _close(res, want, 5e-6)
    _close(out, O.rms(want, 1e-3) * wn, 6e-3 if dtype == "bfloat16" else 1e-5)


# ---- residual rows and products --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("rows,width", [(1, 1), (3, 90), (40, 2304), (2, 4100)])
def test_residual_rows(rows, width, dtype):
    from cacheir_b200 import hybrid_ops as H

    td, tol = DTYPES[dtype][0], 6e-3 if dtype == "bfloat16" else 1e-5
    rng = np.random.default_rng(width)
    y1, y1n = _rand(rng, rows, width, dtype=td)
    y2, y2n = _rand(rng, rows, width, scale=3.0, dtype=td)
    (w1, w1n), (w2, w2n), (w, wn) = (_rand(rng, width, dtype=torch.float32) for _ in range(3))
    table, tn = _rand(rng, 11, width, dtype=td)
    ids = torch.from_numpy(rng.integers(0, 11, rows)).cuda()
    emb = tn[ids.cpu().numpy()]
    for norm in (None, H.RmsNorm(w, 1e-3)):
        def left(x):
            return x if norm is None else O.rms(x, 1e-3) * wn
        res, want = torch.empty((rows, width), device="cuda"), emb * 0.37
        out = torch.empty((rows, width), device="cuda", dtype=td)
        H.scaled_embedding(table, ids, res, 0.37, H.Next(out, norm))
        _close(res, want, 1e-6)
        _close(out, left(want), tol)
        H.residual_add(res, y1, H.Next(out, norm))
        want = want + y1n
        _close(res, want, 1e-6)
        _close(out, left(want), tol)
        H.residual_rms_pair(res, y1, w1, y2, w2, 0.5, 1e-2, H.Next(out, norm))
        want = want + 0.5 * (O.rms(y1n, 1e-2) * w1n + O.rms(y2n, 1e-2) * w2n)
        _close(res, want, 5e-6)
        _close(out, left(want), tol)
        H.scaled_embedding(table, ids, res, 0.37, H.Next(out, norm), accumulate=True)
        want = want + emb * 0.37
        _close(res, want, 5e-6)
        _close(out, left(want), tol)
    H.residual_add(res, y2)
    _close(res, want + y2n, 5e-6)


@pytest.mark.parametrize("t,n,tail,k", [(1, 8, 2, 8), (17, 136, 7, 264), (64, 512, 64, 2048), (130, 250, 3, 72), (520, 1024, 1, 128)])
def test_plain_products_with_a_float_tail(t, n, tail, k):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(t + n)
    x, xn = _rand(rng, t, k)
    w, wn = _rand(rng, n, k, scale=k ** -0.5)
    y = xn @ wn.T
    for epilogue, act in ((H.DENSE_PLAIN, 0), (H.DENSE_SILU, 4)):
        out = torch.full((t, n), 5.0, device="cuda", dtype=torch.bfloat16)
        rest = torch.full((t, tail + 2), 5.0, device="cuda")
        H.dense_gemm(x, w, out, epilogue=epilogue, act_cols=act, tail=rest[:, :tail])
        main = y[:, :n - tail].copy()
        main[:, :act] *= O.sigmoid(main[:, :act])
        _close(out[:, :n - tail], main, 5e-3)
        _close(rest[:, :tail], y[:, n - tail:], 2e-5)
        assert float((out[:, n - tail:] - 5).abs().max()) == 0.0 and float((rest[:, tail:] - 5).abs().max()) == 0.0
