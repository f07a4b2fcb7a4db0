"""Latent attention and the linear recurrence as kernels: ragged batches, pages and slots in any order, portions, windows'
edges with keys that stand out, and sequences much longer than a window or a chunk."""
import numpy as np
import pytest
import torch

from oracle import gutorax as G

pytestmark = pytest.mark.gpu

TYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _bf16(a):
    return torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16)


def make_rows(starts, counts, slots, tables, *, pad=0, pad_segments=0, decode=False):
    """Rows of a step: sequence s brings counts[s] tokens from position starts[s]."""
    from cacheir_b200.hybrid_ops import Rows

    width = max(len(t) for t in tables)
    positions = np.concatenate([np.arange(s, s + n) for s, n in zip(starts, counts)] + [np.zeros(pad)])
    seg = np.concatenate([np.full(n, i) for i, n in enumerate(counts)] + [np.full(pad, -1)])
    cu = np.concatenate([[0], np.cumsum(counts), np.full(pad_segments, sum(counts))])
    table = np.zeros((len(counts) + pad_segments, width))
    for i, t in enumerate(tables):
        table[i, :len(t)] = t
    dev = [torch.from_numpy(np.asarray(a).astype(np.int32)).cuda()
           for a in (positions, seg, cu, table, list(slots) + [0] * pad_segments)]
    return Rows(positions=dev[0], row_seg=dev[1], cu_rows=dev[2], page_table=dev[3], slots=dev[4], decode=decode)


class LatentCase:
    """Sequences with random projections, run through the kernels portion by portion and through the oracle at once."""

    def __init__(self, dtype, heads, dim, rot, vdim, rank, window, lengths, *, page=64, seed=0, sharp=None, rot_dims=None):
        from cacheir_b200 import hybrid_ops as H
        from cacheir_b200.ragged import rotate_half_table

        self.H, self.td = H, TYPES[dtype]
        self.heads, self.dim, self.rot, self.vdim, self.rank, self.window, self.page = heads, dim, rot, vdim, rank, window, page
        self.rot_dims = rot if rot_dims is None else rot_dims
        rng = np.random.default_rng(seed)
        self.scale, self.eps = 0.3, 1e-5
        self.lengths = lengths
        self.down = [_bf16(rng.standard_normal((n, rank + rot))) for n in lengths]
        self.q = [_bf16(rng.standard_normal((n, heads * (dim + rot)))) for n in lengths]
        self.gate = [_bf16(rng.standard_normal((n, heads * vdim))) for n in lengths]
        self.uk, self.uv = _bf16(rng.standard_normal((heads * dim, rank)) * rank ** -0.5), _bf16(rng.standard_normal((heads * vdim, rank)) * rank ** -0.5)
        self.norm = torch.from_numpy(rng.uniform(0.5, 1.5, rank).astype(np.float32))
        self.sink = torch.from_numpy(rng.normal(0, 1, heads).astype(np.float32))
        if sharp is not None:
            sharp(self)
        pages = [(n + page - 1) // page for n in lengths]
        order = rng.permutation(sum(pages) + 3)
        self.tables = np.split(order[:sum(pages)], np.cumsum(pages)[:-1])
        self.num_slots = sum(pages) + 3
        self.pool = torch.full((self.num_slots, page, rank + rot), float("nan"), device="cuda", dtype=self.td)      # leftovers of other owners
        self.table = torch.from_numpy(rotate_half_table(max(lengths) + 1, self.rot_dims, 1000.0)).cuda()

    def oracle(self):
        out = []
        for i in range(len(self.lengths)):
            n, heads, dim, rot = self.lengths[i], self.heads, self.dim, self.rot
            d = self.down[i].double().numpy()
            c = G.rms(d[:, :self.rank], self.eps) * self.norm.double().numpy()
            r = G.rotate_half(d[:, self.rank:], 1000.0, self.rot_dims)
            q = self.q[i].double().numpy().reshape(n, heads, dim + rot)
            q = np.concatenate([q[..., :dim], G.rotate_half(q[..., dim:], 1000.0, self.rot_dims)], -1)
            k = np.concatenate([(c @ self.uk.double().numpy().T).reshape(n, heads, dim), np.broadcast_to(r[:, None], (n, heads, rot))], -1)
            v = (c @ self.uv.double().numpy().T).reshape(n, heads, self.vdim)
            o = G.windowed_sink_attention(q, k, v, self.scale, self.window, self.sink.double().numpy())
            out.append(o.reshape(n, -1) * G.sigmoid(self.gate[i].double().numpy()))
        return out

    def run(self, starts, counts, *, fast, decode=False, pad=0, splits=None):
        H, which = self.H, [i for i, n in enumerate(counts) if n]
        rows = make_rows([starts[i] for i in which], [counts[i] for i in which], range(len(which)), [self.tables[i] for i in which],
                         pad=pad, pad_segments=min(pad, 2), decode=decode)

        def gather(parts, cols):
            t = torch.cat([parts[i][starts[i]:starts[i] + counts[i]] for i in which])
            t = torch.cat([t, torch.zeros((pad, t.shape[1]), dtype=t.dtype)])
            return t.to(self.td).cuda()

        q, down, gate = gather(self.q, 0), gather(self.down, 0), gather(self.gate, 0)
        args = H.latent_args(rows, self.pool, heads=self.heads, dim=self.dim, rot_dim=self.rot, vdim=self.vdim, kv_rank=self.rank,
                             window=self.window, scale=self.scale)
        uk, uv, sink, norm = self.uk.to(self.td).cuda(), self.uv.to(self.td).cuda(), self.sink.cuda(), self.norm.cuda()
        t, width = int(q.shape[0]), self.rank + self.rot
        out = torch.zeros((t, self.heads * self.vdim), device="cuda", dtype=self.td)
        if fast:
            lat = torch.zeros((t, self.heads * width), device="cuda", dtype=self.td)
            H.latent_prepare(args, q, lat[:, self.rank:], q_rot_head_stride=width, table=self.table, rot_dims=self.rot_dims, down=down,
                             norm_weight=norm, eps=self.eps)
            uk_t = uk.view(self.heads, self.dim, self.rank).transpose(1, 2).reshape(self.heads * self.rank, self.dim).contiguous()
            H.dense_gemm(q, uk_t, lat, batch=self.heads, x_batch_cols=self.dim + self.rot, y_batch_cols=width)
            o = torch.zeros((t, self.heads * self.rank), device="cuda", dtype=self.td)
            H.latent_attention(args, lat, sink, o, splits=splits if splits else 1)
            H.dense_gemm(o, uv, out, epilogue=H.DENSE_GATED, batch=self.heads, x_batch_cols=self.rank, gate=gate)
        else:
            H.latent_prepare(args, q, q[:, self.dim:], q_rot_head_stride=self.dim + self.rot, table=self.table, rot_dims=self.rot_dims,
                             down=down, norm_weight=norm, eps=self.eps)
            H.latent_attention_simple(args, q, uk, uv, sink, gate, out)
        parts, row = {}, 0
        for i in which:
            parts[i] = out[row:row + counts[i]].double().cpu().numpy()
            row += counts[i]
        return parts

    def run_schedule(self, schedule, **kwargs):
        """schedule: list of per-sequence token counts; returns the outputs of every sequence, whole."""
        at, got = [0] * len(self.lengths), [[] for _ in self.lengths]
        for counts in schedule:
            for i, part in self.run(at, counts, **kwargs).items():
                got[i].append(part)
            at = [a + n for a, n in zip(at, counts)]
        assert at == list(self.lengths)
        assert self.H.device_status() == 0
        return [np.concatenate(g) for g in got]


def _check(got, want, tol):
    for i, (g, w) in enumerate(zip(got, want)):
        err = np.abs(g - w).max(axis=1) / np.abs(w).max()
        assert np.isfinite(err).all() and err.max() <= tol, (i, int(err.argmax()), float(err.max()))


TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}
#              heads dim rot vdim rank window
LATENT = [(2, 8, 8, 16, 8, 70), (3, 16, 8, 24, 48, 5), (1, 8, 16, 16, 16, 64), (17, 16, 64, 32, 128, 65), (40, 32, 16, 16, 256, 130), (32, 64, 64, 64, 512, 200),
          (65, 8, 8, 8, 32, 40)]


@pytest.mark.parametrize("shape", LATENT)
@pytest.mark.parametrize("form", ["simple32", "simple16", "fast"])
def test_latent_attention_prompts_and_portions(shape, form):
    dtype = "float32" if form == "simple32" else "bfloat16"
    lengths = (150, 1, 67)
    schedules = [[lengths], [(63, 1, 2), (2, 0, 30), (64, 0, 0), (21, 0, 35)]]
    want = None
    for schedule in schedules:
        case = LatentCase(dtype, *shape, lengths)
        want = want or case.oracle()
        _check(case.run_schedule(schedule, fast=form == "fast", pad=3), want, TOL[dtype])


@pytest.mark.parametrize("shape", LATENT)
@pytest.mark.parametrize("splits", [1, 2, 8])
def test_latent_attention_decodes_what_prompts_give(shape, splits):
    lengths = (140, 140)
    case = LatentCase("bfloat16", *shape, lengths)
    want = case.oracle()
    got = case.run((0, 0), (100, 100), fast=True)
    _check([got[0], got[1]], [w[:100] for w in want], TOL["bfloat16"])
    for pos in range(100, 140):
        step = case.run((pos, pos), (1, 1), fast=True, decode=True, splits=splits)
        _check([step[0], step[1]], [w[pos:pos + 1] for w in want], 2.5e-2 * max(1.0, np.abs(want[0]).max() / np.abs(want[0][pos]).max()))
    assert case.H.device_status() == 0


@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 128, 129])
@pytest.mark.parametrize("form", ["simple32", "fast", "decode"])
def test_window_edges_with_keys_that_stand_out(window, form):
    """Position p asks for one key `gap` tokens back so strongly that it takes nearly all weight: inside the window it is
    read, one token further away it is gone and the sink takes over."""
    n = 300
    gaps = {150 + window: window - 1, 151 + window: window, 140: window - 1, 141: window}

    def sharp(case):
        for p, gap in gaps.items():
            j = p - gap
            if j < 0:
                continue
            case.q[0].view(n, case.heads, -1)[p, :, case.dim:] = 0
            c = case.down[0][j, :case.rank].double().numpy()
            key = (case.uk.double().numpy() @ (G.rms(c, case.eps) * case.norm.double().numpy())).reshape(case.heads, case.dim)
            case.q[0].view(n, case.heads, -1)[p, :, :case.dim] = _bf16(key * 40.0 / (0.3 * (key ** 2).sum(-1, keepdims=True)))

    dtype = "float32" if form == "simple32" else "bfloat16"
    case = LatentCase(dtype, 2, 32, 16, 32, 64, window, (n,), sharp=sharp)
    want = case.oracle()[0]
    if form == "decode":
        first = min(p for p in gaps if gaps[p] <= p)
        got = [case.run((0,), (first,), fast=True)[0]]
        got += [case.run((p,), (1,), fast=True, decode=True, splits=1 + p % 3)[0] for p in range(first, n)]
        got = np.concatenate(got)
    else:
        got = case.run_schedule([(n,)], fast=form == "fast")[0]
    scale = np.abs(want).max()
    assert np.abs(got - want).max() / scale <= (1e-4 if dtype == "float32" else 6e-2)
    # the rows really hinge on the edge: with a window one token shorter the asked key is out of sight
    case.window = window - 1
    if window > 1:
        moved = case.oracle()[0]
        for p, gap in gaps.items():
            if 0 <= p - gap and gap == window - 1:
                assert np.abs(moved[p] - want[p]).max() > 0.15 * np.abs(want[p]).max()


def test_shared_cache_layer_appends_nothing():
    case = LatentCase("bfloat16", 2, 16, 16, 16, 32, 20, (50,))
    case.run_schedule([(50,)], fast=True)
    before = case.pool.clone()
    H = case.H
    rows = make_rows([49], [1], [0], [case.tables[0]])
    args = H.latent_args(rows, case.pool, heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=32, window=20, scale=1.0)
    q = case.q[0][49:50].cuda()
    turned = torch.zeros((1, 2 * 16), device="cuda", dtype=torch.bfloat16)
    H.latent_prepare(args, q, turned, q_rot_head_stride=16, table=case.table, rot_dims=16)
    assert torch.equal(before.view(torch.int16), case.pool.view(torch.int16))
    want = G.rotate_half(np.concatenate([np.zeros((49, 2, 16)), case.q[0][49:50].double().numpy().reshape(1, 2, 32)[..., 16:]]), 1000.0, 16)[49]
    np.testing.assert_allclose(turned.double().cpu().numpy().reshape(2, 16), want, atol=2e-2)


# ---- recurrence -----------------------------------------------------------------------------------------------------------
class RecurrenceCase:
    def __init__(self, dtype, heads, dim, vdim, lengths, *, decay=None, seed=0):
        from cacheir_b200 import hybrid_ops as H

        self.H, self.td, self.heads, self.dim, self.vdim, self.lengths = H, TYPES[dtype], heads, dim, vdim, lengths
        rng = np.random.default_rng(seed)
        self.decay = [1.0 - 2.0 ** -(h % 9) for h in range(heads)] if decay is None else decay       # 0, 0.5, 0.75 ... close to 1
        cols = heads * (2 * dim + vdim)
        self.stride = (cols + 7) // 8 * 8 + 8
        self.qkv = [_bf16(rng.standard_normal((n, self.stride)) * 0.7) for n in lengths]
        self.powers = H.decay_powers(self.decay, "cuda")
        self.slots = rng.permutation(len(lengths) + 2)[:len(lengths)]
        self.state = torch.full((len(lengths) + 2, heads, dim, vdim), 1e6, device="cuda")            # leftovers of other owners

    def _split(self, a):
        h, d, e = self.heads, self.dim, self.vdim
        return a[:, :h * d], a[:, h * d:2 * h * d], a[:, 2 * h * d:h * (2 * d + e)]

    def oracle(self):
        outs = []
        for a in self.qkv:
            q, k, v = self._split(a.double().numpy())
            n = q.shape[0]
            outs.append(G.decayed_outer_recurrence(q.reshape(n, self.heads, -1), k.reshape(n, self.heads, -1), v.reshape(n, self.heads, -1),
                                                   [float(p) for p in self.powers[:, 1].double().cpu()]))
        return outs

    def run(self, starts, counts, form, *, pad=0):
        H, which = self.H, [i for i, n in enumerate(counts) if n]
        rows = make_rows([starts[i] for i in which], [counts[i] for i in which], [self.slots[i] for i in which], [[0]] * len(which),
                         pad=pad, pad_segments=min(pad, 2), decode=form == "step")
        x = torch.cat([self.qkv[i][starts[i]:starts[i] + counts[i]] for i in which] + [torch.zeros((pad, self.stride), dtype=torch.bfloat16)])
        x = x.to(self.td).cuda()
        q, k, v = self._split(x)
        out = torch.zeros((x.shape[0], self.heads * self.vdim), device="cuda", dtype=self.td)
        args = H.recurrence_args(rows, q, k, v, self.powers, self.state, out, heads=self.heads, dim=self.dim, vdim=self.vdim)
        if form == "chunked":
            need = H.recurrence_workspace_bytes(rows.rows, rows.segments, self.heads, self.dim, self.vdim)
            ws = torch.full((need,), 0xFF, device="cuda", dtype=torch.uint8) if need else None      # NaN patterns: nothing may be read unwritten
            H.recurrence_chunked(args, ws)
        else:
            (H.recurrence_step if form == "step" else H.recurrence_simple)(args)
        parts, row = {}, 0
        for i in which:
            parts[i] = out[row:row + counts[i]].double().cpu().numpy()
            row += counts[i]
        return parts

    def run_schedule(self, schedule, **kwargs):
        at, got = [0] * len(self.lengths), [[] for _ in self.lengths]
        for form, counts in schedule:
            for i, part in self.run(at, counts, form, **kwargs).items():
                got[i].append(part)
            at = [a + n for a, n in zip(at, counts)]
        assert at == list(self.lengths)
        return [np.concatenate(g) for g in got]

    def check(self, got, out_tol, state_tol):
        for i, (out, state) in enumerate(self.oracle()):
            want = out.reshape(out.shape[0], -1)
            for h in range(self.heads):      # head by head: their sizes differ by orders of magnitude
                cols = slice(h * self.vdim, (h + 1) * self.vdim)
                err = np.abs(got[i][:, cols] - want[:, cols]).max(axis=1) / np.abs(want[:, cols]).max()
                assert np.isfinite(err).all() and err.max() <= out_tol, (i, h, int(err.argmax()), float(err.max()))
                s = self.state[self.slots[i], h].double().cpu().numpy()
                assert np.abs(s - state[h]).max() / np.abs(state[h]).max() <= state_tol, (i, h)


RECURRENT = [(3, 32, 72), (9, 16, 8), (2, 128, 128), (4, 48, 64), (1, 64, 200), (2, 112, 24)]


@pytest.mark.parametrize("shape", RECURRENT)
@pytest.mark.parametrize("form", ["chunked", "simple"])
def test_recurrence_prompts(shape, form):
    case = RecurrenceCase("bfloat16", *shape, (70, 1, 64, 300, 2))
    case.check(case.run_schedule([(form, case.lengths)], pad=5), 6e-3, 3e-5)


@pytest.mark.parametrize("shape", RECURRENT + [(2, 5, 7), (1, 1, 1), (3, 130, 33)])
def test_recurrence_in_32_bit(shape):
    case = RecurrenceCase("float32", *shape, (40, 1, 130))
    step = "step" if shape[2] % 4 == 0 else "simple"
    plan = [("simple", (17, 0, 64)), ("simple", (20, 0, 2)), ("simple", (2, 1, 63)), (step, (1, 0, 1))]
    case.check(case.run_schedule(plan), 1e-5, 1e-5)


@pytest.mark.parametrize("shape", RECURRENT)
def test_recurrence_portions_and_decoding_carry_the_state(shape):
    case = RecurrenceCase("bfloat16", *shape, (700, 90))
    plan = [("chunked", (63, 2)), ("chunked", (2, 0)), ("step", (1, 1)), ("chunked", (513, 64)), ("chunked", (2, 2)), ("simple", (98, 3))]
    plan += [("step", (1, 1)), ("chunked", (20, 0))] + [("step", (0, 1))] * 16 + [("chunked", (0, 1))]
    case.check(case.run_schedule(plan), 6e-3, 3e-5)


def test_recurrence_pieces_with_slow_decay_remember_the_first_token():
    """2 000 tokens of which only the first has a key: everything later reads it through the carried state."""
    case = RecurrenceCase("bfloat16", 2, 32, 64, (2000,), decay=[0.9995, 1.0])
    k = case.qkv[0][:, 2 * 32:4 * 32]
    k[1:] = 0
    want = case.oracle()[0][0].reshape(2000, -1)
    assert np.abs(want[-1, :64]).max() > 0.1 * np.abs(want[0, :64]).max()
    got = case.run_schedule([("chunked", (2000,))])[0]
    err = np.abs(got - want).max(axis=1) / np.abs(want).max()
    assert err.max() <= 6e-3
