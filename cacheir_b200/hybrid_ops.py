"""Torch-tensor wrappers over the C ABI of the ragged families (include/cacheir_b200_ragged.h, cacheir_b200_hybrid.h,
cacheir_b200_recurrence.h).

Same rules as `ops`: validate, pass device pointers on the current stream, raise on a non-zero status. The residual
stream and every norm parameter are float32; activations are float32 or bfloat16.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from ._lib import DenseArgs, LatentArgs, RecurrenceArgs, check
from .ops import _ptr, _require_cuda, _stream, dtype_code

NEXT_NONE, NEXT_COPY, NEXT_DYT, NEXT_RMS, NEXT_LAYER = range(5)
(DENSE_PLAIN, DENSE_F32, DENSE_SILU, DENSE_GEGLU, DENSE_GATED, DENSE_RESIDUAL, DENSE_GELU_EMBED, DENSE_SWIGLU,
 DENSE_CLAMPED_GLU, DENSE_RELU2) = range(10)
GLU_EPILOGUES = {"gelu_tanh": DENSE_GEGLU, "silu": DENSE_SWIGLU, "clamped": DENSE_CLAMPED_GLU}
RECURRENCE_POWERS = 65


@dataclass
class DynamicTanh:
    """tanh(alpha * x) * weight + bias; weight and bias float32 on the device."""

    weight: torch.Tensor
    bias: torch.Tensor
    alpha: float


@dataclass
class RmsNorm:
    """x / sqrt(mean(x^2) + eps) * weight; weight float32 on the device."""

    weight: torch.Tensor
    eps: float


@dataclass
class LayerNorm:
    """(x - mean) / sqrt(variance + eps) * weight; weight float32 on the device."""

    weight: torch.Tensor
    eps: float


@dataclass
class Next:
    """What a kernel that finishes the residual leaves in `out`: the residual itself or a norm of it."""

    out: torch.Tensor
    norm: DynamicTanh | RmsNorm | LayerNorm | None = None


@dataclass
class Rows:
    """The rows of a ragged step (see the header for the meaning of the tensors)."""

    positions: torch.Tensor
    row_seg: torch.Tensor
    cu_rows: torch.Tensor
    page_table: torch.Tensor
    slots: torch.Tensor
    decode: bool

    @property
    def rows(self) -> int:
        return int(self.positions.numel())

    @property
    def segments(self) -> int:
        return int(self.cu_rows.numel()) - 1


def _next(nx: Next | None) -> tuple:
    if nx is None:
        return (NEXT_NONE, None, None, 0.0, None)
    if nx.norm is None:
        return (NEXT_COPY, None, None, 0.0, nx.out.data_ptr())
    if isinstance(nx.norm, (RmsNorm, LayerNorm)):
        _f32(nx.norm.weight)
        return (NEXT_RMS if isinstance(nx.norm, RmsNorm) else NEXT_LAYER, nx.norm.weight.data_ptr(), None, float(nx.norm.eps), nx.out.data_ptr())
    return (NEXT_DYT, nx.norm.weight.data_ptr(), nx.norm.bias.data_ptr(), float(nx.norm.alpha), nx.out.data_ptr())


def _f32(*tensors: torch.Tensor) -> None:
    for t in tensors:
        if t.dtype != torch.float32 or not t.is_contiguous():
            raise ValueError("norm parameters and the residual stream are contiguous float32 tensors")


def dense_supported(k: int, w_stride: int, x_stride: int, *, dtype: torch.dtype, batch: int = 1, x_batch_cols: int = 0) -> bool:
    """Can the tensor-core GEMM take this product?"""
    return dtype == torch.bfloat16 and bool(_lib.load_group("ragged").cacheir_b200_dense_supported(k, w_stride, x_stride, batch, x_batch_cols))


def dense_gemm(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor | None = None, *, epilogue: int = DENSE_PLAIN,
               batch: int = 1, x_batch_cols: int = 0, y_batch_cols: int | None = None, act_cols: int = 0, gate: torch.Tensor | None = None,
               residual: torch.Tensor | None = None, norm: DynamicTanh | None = None, nx: Next | None = None,
               ids: torch.Tensor | None = None, table: torch.Tensor | None = None, table_col: int = 0,
               bias: torch.Tensor | None = None, limit: float = 0.0, tail: torch.Tensor | None = None) -> None:
    """Tensor-core Y = f(X W^T + bias). x [T, >=K] and w [N, K] bf16 with dense rows. `batch` > 1: w [batch*N, K], entry z
    reads x columns from z*x_batch_cols and writes output columns from z*y_batch_cols (default z*N). `tail` (plain, SiLU and
    paired epilogues): the last columns of the product go there as float32."""
    _require_cuda(x, w, out, gate, residual, ids, table)
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or x.stride(1) != 1 or w.stride(1) != 1:
        raise ValueError("dense_gemm takes bf16 x and w with dense rows")
    a = DenseArgs()
    a.x, a.w, a.T, a.K = x.data_ptr(), w.data_ptr(), int(x.shape[0]), int(w.shape[1])
    a.N = int(w.shape[0]) // batch
    a.batch, a.w_batch_rows, a.x_batch_cols, a.y_batch_cols = batch, a.N, x_batch_cols, a.N if y_batch_cols is None else y_batch_cols
    a.w_stride, a.x_stride, a.epilogue = w.stride(0), x.stride(0), epilogue
    if epilogue == DENSE_RESIDUAL:
        if residual is None or norm is None or tuple(residual.shape) != (a.T, a.N):
            raise ValueError("the residual epilogue needs the [T, N] residual and its norm")
        _f32(residual, norm.weight, norm.bias)
        a.residual, a.norm_w, a.norm_b, a.norm_alpha = residual.data_ptr(), norm.weight.data_ptr(), norm.bias.data_ptr(), float(norm.alpha)
        a.next_mode, a.next_w, a.next_b, a.next_alpha, a.next_out = _next(nx)
        if nx is not None and (tuple(nx.out.shape) != (a.T, a.N) or nx.out.dtype != torch.bfloat16 or not nx.out.is_contiguous()):
            raise ValueError("the next operator's input must be a contiguous bf16 [T, N] tensor")
    else:
        paired = epilogue in GLU_EPILOGUES.values()
        if tail is not None:
            if not (paired or epilogue in (DENSE_PLAIN, DENSE_SILU)) or tail.dtype != torch.float32 or tail.stride(1) != 1 or int(tail.shape[0]) != a.T:
                raise ValueError("tail is a float32 [T, columns] tensor of a plain, SiLU or paired epilogue")
            a.tail, a.tail_cols, a.tail_stride = tail.data_ptr(), int(tail.shape[1]), tail.stride(0)
        cols = (a.N - a.tail_cols) // 2 if paired else a.y_batch_cols * (batch - 1) + a.N - a.tail_cols
        want = torch.float32 if epilogue == DENSE_F32 else torch.bfloat16
        if out is None or out.dtype != want or int(out.shape[0]) != a.T or int(out.shape[1]) < cols or out.stride(1) != 1:
            raise ValueError("out must be [T, N] of the epilogue's type with dense rows")
        a.y, a.y_stride, a.act_cols = out.data_ptr(), out.stride(0), act_cols
    a.limit = float(limit)
    if bias is not None:
        _f32(bias)
        if batch != 1 or bias.numel() != a.N:
            raise ValueError("bias has one entry per output column")
        a.bias = bias.data_ptr()
    if epilogue == DENSE_GATED:
        if gate is None or gate.dtype != torch.bfloat16 or gate.stride(1) != 1 or int(gate.shape[1]) < a.N * batch:
            raise ValueError("the gated epilogue needs a bf16 gate per output column")
        a.gate, a.gate_stride = gate.data_ptr(), gate.stride(0)
    if epilogue == DENSE_GELU_EMBED:
        if ids is None or table is None or ids.dtype != torch.int64 or int(table.shape[1]) < table_col + a.N:
            raise ValueError("the embedding epilogue needs int64 ids and a table with a part for every output column")
        a.ids, a.table, a.table_stride, a.table_col, a.vocab = ids.data_ptr(), table.data_ptr(), table.stride(0), table_col, int(table.shape[0])
    check(_lib.load_group("ragged").cacheir_b200_dense_gemm(ctypes.byref(a), _stream()), "dense_gemm")


def dense_simple(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, batch: int = 1, x_batch_cols: int = 0,
                 bias: torch.Tensor | None = None) -> torch.Tensor:
    """The plain product in float32 arithmetic on the CUDA cores, any extents (see dense_gemm for `batch`)."""
    _require_cuda(x, w, out, bias)
    n, k = int(w.shape[0]) // batch, int(w.shape[1])
    if x.dtype != w.dtype or x.stride(1) != 1 or w.stride(1) != 1 or out.stride(1) != 1 or int(out.shape[1]) < n * batch:
        raise ValueError("dense_simple takes x, w of one type with dense rows and out [T, N]")
    check(_lib.load_group("ragged").cacheir_b200_dense_simple(
        x.data_ptr(), w.data_ptr(), out.data_ptr(), int(x.shape[0]), n, k, batch, n, x_batch_cols, n, w.stride(0), x.stride(0),
        out.stride(0), _ptr(bias), dtype_code(x.dtype), dtype_code(out.dtype), _stream()), "dense_simple")
    return out


def scaled_embedding(table: torch.Tensor, ids: torch.Tensor, residual: torch.Tensor, scale: float, nx: Next | None = None, *,
                     accumulate: bool = False) -> None:
    """residual = table[ids] * scale, or (`accumulate`) that much more."""
    _require_cuda(table, ids, residual)
    _f32(residual)
    if ids.dtype != torch.int64 or not table.is_contiguous() or residual.shape[1] != table.shape[1]:
        raise ValueError("scaled_embedding expects int64 ids and a contiguous [vocab, width] table")
    check(_lib.load_group("ragged").cacheir_b200_scaled_embedding(
        table.data_ptr(), ids.data_ptr(), residual.data_ptr(), int(residual.shape[0]), int(table.shape[1]), int(table.shape[0]),
        float(scale), int(accumulate), *_next(nx), dtype_code(table.dtype), _stream()), "scaled_embedding")


def dyt_rows(residual: torch.Tensor, norm: DynamicTanh, out: torch.Tensor, row_index: torch.Tensor | None = None) -> torch.Tensor:
    """out[j] = dynamic tanh of residual row row_index[j] (row j without an index)."""
    _require_cuda(residual, out, row_index)
    _f32(residual, norm.weight, norm.bias)
    check(_lib.load_group("ragged").cacheir_b200_dyt_rows(
        residual.data_ptr(), _ptr(row_index), norm.weight.data_ptr(), norm.bias.data_ptr(), float(norm.alpha), out.data_ptr(),
        int(out.shape[0]), int(out.shape[1]), dtype_code(out.dtype), _stream()), "dyt_rows")
    return out


def rms_rows(residual: torch.Tensor, weight: torch.Tensor, eps: float, out: torch.Tensor, row_index: torch.Tensor | None = None) -> torch.Tensor:
    """out[j] = rms_norm(residual row row_index[j]) * weight (row j without an index)."""
    _require_cuda(residual, weight, out, row_index)
    _f32(residual, weight)
    check(_lib.load_group("ragged").cacheir_b200_rms_rows(
        residual.data_ptr(), _ptr(row_index), weight.data_ptr(), float(eps), out.data_ptr(), int(out.shape[0]), int(out.shape[1]),
        dtype_code(out.dtype), _stream()), "rms_rows")
    return out


def residual_dyt(residual: torch.Tensor, y: torch.Tensor, norm: DynamicTanh, nx: Next | None = None) -> None:
    _require_cuda(residual, y)
    _f32(residual, norm.weight, norm.bias)
    if y.shape != residual.shape or not y.is_contiguous():
        raise ValueError("y must be a contiguous tensor of the residual's shape")
    check(_lib.load_group("ragged").cacheir_b200_residual_dyt(
        residual.data_ptr(), y.data_ptr(), norm.weight.data_ptr(), norm.bias.data_ptr(), float(norm.alpha), int(y.shape[0]),
        int(y.shape[1]), *_next(nx), dtype_code(y.dtype), _stream()), "residual_dyt")


def layer_norm_rows(residual: torch.Tensor, weight: torch.Tensor, eps: float, out: torch.Tensor, row_index: torch.Tensor | None = None) -> torch.Tensor:
    """out[j] = layer norm of residual row row_index[j] (row j without an index) * weight."""
    _require_cuda(residual, weight, out, row_index)
    _f32(residual, weight)
    check(_lib.load_group("ragged").cacheir_b200_layer_norm_rows(
        residual.data_ptr(), _ptr(row_index), weight.data_ptr(), float(eps), out.data_ptr(), int(out.shape[0]), int(out.shape[1]),
        dtype_code(out.dtype), _stream()), "layer_norm_rows")
    return out


def join_embedding(residual: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """out [rows, 2*width] = (residual | table[ids])"""
    _require_cuda(residual, table, ids, out)
    _f32(residual)
    if ids.dtype != torch.int64 or not table.is_contiguous() or residual.shape[1] != table.shape[1] or table.dtype != out.dtype \
            or tuple(out.shape) != (residual.shape[0], 2 * residual.shape[1]) or not out.is_contiguous():
        raise ValueError("join_embedding expects int64 ids, a contiguous [vocab, width] table and a contiguous [rows, 2*width] output")
    check(_lib.load_group("ragged").cacheir_b200_join_embedding(
        residual.data_ptr(), table.data_ptr(), ids.data_ptr(), out.data_ptr(), int(residual.shape[0]), int(table.shape[1]), int(table.shape[0]),
        dtype_code(out.dtype), _stream()), "join_embedding")
    return out


def residual_add(residual: torch.Tensor, y: torch.Tensor, nx: Next | None = None, scale: torch.Tensor | None = None) -> None:
    """residual += y, or y * scale column by column"""
    _require_cuda(residual, y, scale)
    _f32(residual, *([] if scale is None else [scale]))
    if y.shape != residual.shape or not y.is_contiguous() or (scale is not None and scale.numel() != residual.shape[1]):
        raise ValueError("y must be a contiguous tensor of the residual's shape, scale have an entry per column")
    check(_lib.load_group("ragged").cacheir_b200_residual_add(
        residual.data_ptr(), y.data_ptr(), _ptr(scale), int(y.shape[0]), int(y.shape[1]), *_next(nx), dtype_code(y.dtype), _stream()), "residual_add")


def residual_rms_pair(residual: torch.Tensor, y1: torch.Tensor, w1: torch.Tensor, y2: torch.Tensor, w2: torch.Tensor, factor: float, eps: float,
                      nx: Next | None = None) -> None:
    """residual += factor * (rms_norm(y1) * w1 + rms_norm(y2) * w2)"""
    _require_cuda(residual, y1, y2, w1, w2)
    _f32(residual, w1, w2)
    if any(y.shape != residual.shape or not y.is_contiguous() or y.dtype != y1.dtype for y in (y1, y2)):
        raise ValueError("y1 and y2 must be contiguous tensors of the residual's shape and one type")
    check(_lib.load_group("ragged").cacheir_b200_residual_rms_pair(
        residual.data_ptr(), y1.data_ptr(), w1.data_ptr(), y2.data_ptr(), w2.data_ptr(), float(factor), float(eps), int(y1.shape[0]),
        int(y1.shape[1]), *_next(nx), dtype_code(y1.dtype), _stream()), "residual_rms_pair")


def residual_rms(residual: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float, nx: Next | None = None) -> None:
    """residual += rms_norm(y) * weight"""
    _require_cuda(residual, y, weight)
    _f32(residual, weight)
    if y.shape != residual.shape or not y.is_contiguous():
        raise ValueError("y must be a contiguous tensor of the residual's shape")
    check(_lib.load_group("ragged").cacheir_b200_residual_rms(
        residual.data_ptr(), y.data_ptr(), weight.data_ptr(), float(eps), int(y.shape[0]), int(y.shape[1]), *_next(nx),
        dtype_code(y.dtype), _stream()), "residual_rms")


def gated_rms(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, eps: float, out: torch.Tensor) -> torch.Tensor:
    """out = rms_norm(o) * weight * sigmoid(gate); gate rows may be a strided view."""
    _require_cuda(o, gate, weight, out)
    _f32(weight)
    if not o.is_contiguous() or not out.is_contiguous() or gate.stride(1) != 1 or gate.shape != o.shape or out.shape != o.shape:
        raise ValueError("gated_rms expects contiguous o and out and a gate of their shape")
    check(_lib.load_group("ragged").cacheir_b200_gated_rms(
        o.data_ptr(), gate.data_ptr(), gate.stride(0), weight.data_ptr(), float(eps), out.data_ptr(), int(o.shape[0]), int(o.shape[1]),
        dtype_code(o.dtype), _stream()), "gated_rms")
    return out


def gated_parts_rms(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, eps: float, out: torch.Tensor, *, parts: int,
                    gate_first: bool) -> torch.Tensor:
    """Norm in equal parts with a silu gate, before the norm or behind it; weight per column of a row, or of a part."""
    _require_cuda(o, gate, weight, out)
    _f32(weight)
    cols = int(o.shape[1])
    if not o.is_contiguous() or not out.is_contiguous() or gate.stride(1) != 1 or gate.shape != o.shape or out.shape != o.shape or cols % parts:
        raise ValueError("gated_parts_rms expects contiguous o and out, a gate of their shape and equal parts")
    if weight.numel() not in (cols, cols // parts):
        raise ValueError("the weight has an entry per column of a row or of a part")
    check(_lib.load_group("ragged").cacheir_b200_gated_parts_rms(
        o.data_ptr(), gate.data_ptr(), gate.stride(0), weight.data_ptr(), int(weight.numel() != cols), int(gate_first), float(eps), out.data_ptr(),
        int(o.shape[0]), cols, int(parts), dtype_code(o.dtype), _stream()), "gated_parts_rms")
    return out


def glu_pairs(y: torch.Tensor, out: torch.Tensor, epilogue: int = DENSE_GEGLU, limit: float = 0.0) -> torch.Tensor:
    """y [T, 2*ff] with columns alternating gate, up; out as the paired epilogue leaves it."""
    _require_cuda(y, out)
    if not y.is_contiguous() or not out.is_contiguous() or y.shape[1] != 2 * out.shape[1]:
        raise ValueError("glu_pairs expects contiguous [T, 2*ff] and [T, ff]")
    check(_lib.load_group("ragged").cacheir_b200_glu_pairs(y.data_ptr(), out.data_ptr(), int(out.shape[0]), int(out.shape[1]), int(epilogue),
                                                           float(limit), dtype_code(y.dtype), _stream()), "glu_pairs")
    return out


def gelu_embed(g: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, table_col: int, out: torch.Tensor) -> torch.Tensor:
    _require_cuda(g, ids, table, out)
    if not g.is_contiguous() or not out.is_contiguous() or table.stride(1) != 1 or int(table.shape[1]) < table_col + int(g.shape[1]):
        raise ValueError("gelu_embed expects contiguous g and out and a table with a part for every column")
    check(_lib.load_group("ragged").cacheir_b200_gelu_embed(
        g.data_ptr(), ids.data_ptr(), table.data_ptr(), table.stride(0), int(table_col), out.data_ptr(), int(g.shape[0]),
        int(g.shape[1]), int(table.shape[0]), dtype_code(g.dtype), _stream()), "gelu_embed")
    return out


def silu_cols(y: torch.Tensor, cols: int) -> torch.Tensor:
    _require_cuda(y)
    check(_lib.load_group("ragged").cacheir_b200_silu_cols(y.data_ptr(), int(y.shape[0]), y.stride(0), int(cols), dtype_code(y.dtype), _stream()),
          "silu_cols")
    return y


def relu2_cols(y: torch.Tensor, cols: int) -> torch.Tensor:
    _require_cuda(y)
    check(_lib.load_group("ragged").cacheir_b200_relu2_cols(y.data_ptr(), int(y.shape[0]), y.stride(0), int(cols), dtype_code(y.dtype), _stream()),
          "relu2_cols")
    return y


# ---- latent attention ------------------------------------------------------------------------------------------------
def latent_args(rows: Rows, pool: torch.Tensor, *, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, window: int,
                scale: float) -> LatentArgs:
    """pool: [slots, page, kv_rank + rot_dim]."""
    if pool.dim() != 3 or int(pool.shape[2]) != kv_rank + rot_dim or not pool.is_contiguous():
        raise ValueError("the latent pool must be a contiguous [slots, page, kv_rank + rot_dim] tensor")
    a = LatentArgs()
    a.positions, a.row_seg, a.cu_rows = rows.positions.data_ptr(), rows.row_seg.data_ptr(), rows.cu_rows.data_ptr()
    a.page_table, a.rows, a.segments = rows.page_table.data_ptr(), rows.rows, rows.segments
    a.max_pages, a.page_size, a.num_slots = int(rows.page_table.shape[1]), int(pool.shape[1]), int(pool.shape[0])
    a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.window, a.scale = heads, dim, rot_dim, vdim, kv_rank, window, float(scale)
    a.pool, a.dtype, a.decode = pool.data_ptr(), dtype_code(pool.dtype), int(rows.decode)
    return a


def latent_prepare(a: LatentArgs, q: torch.Tensor, q_rot: torch.Tensor, *, q_rot_head_stride: int, table: torch.Tensor, rot_dims: int,
                   down: torch.Tensor | None = None, norm_weight: torch.Tensor | None = None, eps: float = 0.0) -> None:
    """Append one cache row per token (unless `down` is None) and turn the queries' rotated part into `q_rot`, a tensor
    whose first element is row 0, head 0's first rotated entry."""
    _require_cuda(q, q_rot, table, down, norm_weight)
    check(_lib.load_group("hybrid").cacheir_b200_latent_prepare(
        ctypes.byref(a), _ptr(down), 0 if down is None else down.stride(0), _ptr(norm_weight), float(eps), q.data_ptr(), q.stride(0),
        q_rot.data_ptr(), q_rot.stride(0), int(q_rot_head_stride), table.data_ptr(), int(table.shape[0]), int(rot_dims), _stream()),
        "latent_prepare")


def latent_attention_simple(a: LatentArgs, q: torch.Tensor, uk: torch.Tensor, uv: torch.Tensor, sink: torch.Tensor, gate: torch.Tensor,
                            out: torch.Tensor) -> torch.Tensor:
    _require_cuda(q, uk, uv, sink, gate, out)
    _f32(sink)
    check(_lib.load_group("hybrid").cacheir_b200_latent_attention_simple(
        ctypes.byref(a), q.data_ptr(), q.stride(0), uk.data_ptr(), uv.data_ptr(), sink.data_ptr(), gate.data_ptr(), gate.stride(0),
        out.data_ptr(), _stream()), "latent_attention_simple")
    return out


def latent_attention_supported(kv_rank: int, rot_dim: int, page_size: int, dtype: torch.dtype) -> bool:
    return bool(_lib.load_group("hybrid").cacheir_b200_latent_attention_supported(kv_rank, rot_dim, page_size, dtype_code(dtype)))


def latent_attention_splits(rows: int, heads: int, window: int, max_pages: int, page_size: int) -> int:
    return int(_lib.load_group("hybrid").cacheir_b200_latent_attention_splits(rows, heads, window, max_pages, page_size))


def latent_attention(a: LatentArgs, q: torch.Tensor, sink: torch.Tensor, out: torch.Tensor, *, splits: int = 1) -> torch.Tensor:
    """q [T, heads*(kv_rank + rot_dim)] in latent space, out [T, heads*kv_rank], both dense bf16."""
    _require_cuda(q, sink, out)
    _f32(sink)
    if not q.is_contiguous() or not out.is_contiguous():
        raise ValueError("latent_attention expects contiguous q and out")
    check(_lib.load_group("hybrid").cacheir_b200_latent_attention(
        ctypes.byref(a), q.data_ptr(), sink.data_ptr(), out.data_ptr(), int(splits), _stream()), "latent_attention")
    return out


# ---- linear recurrence -------------------------------------------------------------------------------------------------
def decay_powers(decay, device: torch.device | str) -> torch.Tensor:
    """[heads, 65] float32: decay^0 .. decay^64, evaluated in double precision."""
    d = torch.tensor([float(v) for v in decay], dtype=torch.float64)
    e = torch.arange(RECURRENCE_POWERS, dtype=torch.float64)
    return torch.pow(d[:, None], e[None, :]).to(torch.float32).contiguous().to(device)


def recurrence_args(rows: Rows, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, powers: torch.Tensor | None, state: torch.Tensor,
                    out: torch.Tensor, *, heads: int, dim: int, vdim: int,
                    gated: tuple[torch.Tensor, torch.Tensor, torch.Tensor | None] | None = None, q_scale: float = 1.0, key_heads: int | None = None,
                    skip: torch.Tensor | None = None, memory: bool = True) -> RecurrenceArgs:
    """q, k [T, key_heads*dim] (by default as many heads as v) and v [T, heads*vdim] with one common row stride. Constant decays:
    state [slots, heads, dim, vdim] float32. Without `powers` the recurrence is gated: `gated` = (log_decay, log_take, normaliser),
    [T, heads] float32 each (not needed by the step forms), and state [slots, memory_state_size(...)], or without `memory` (no
    normaliser) rows of any length that begin with [heads, dim, vdim]. `skip` [heads]: o += skip * v."""
    _require_cuda(q, k, v, powers, state, out, skip)
    given = [] if gated is None else [t for t in gated if t is not None]
    _f32(state, *([] if powers is None else [powers]), *given, *([] if skip is None else [skip]))
    if not (q.stride(0) == k.stride(0) == v.stride(0)) or q.stride(1) != 1 or k.stride(1) != 1 or v.stride(1) != 1:
        raise ValueError("q, k and v must share one row stride and have dense rows")
    if not out.is_contiguous() or (powers is not None and (tuple(state.shape[1:]) != (heads, dim, vdim) or tuple(powers.shape) != (heads, RECURRENCE_POWERS))):
        raise ValueError("state must be [slots, heads, dim, vdim], powers [heads, 65] and out contiguous")
    if powers is None and memory and tuple(state.shape[1:]) != (memory_state_size(heads, dim, vdim),):
        raise ValueError("a gated recurrence's state must be [slots, memory_state_size]")
    if state.stride(0) < heads * dim * vdim or (key_heads is not None and heads % key_heads) or (skip is not None and skip.numel() != heads):
        raise ValueError("a state slot must hold [heads, dim, vdim], key heads divide the heads, skip has an entry per head")
    if any(tuple(t.shape) != (rows.rows, heads) for t in given):
        raise ValueError("log_decay, log_take and normaliser are [rows, heads]")
    a = RecurrenceArgs()
    a.positions, a.cu_rows, a.slots = rows.positions.data_ptr(), rows.cu_rows.data_ptr(), rows.slots.data_ptr()
    a.rows, a.segments, a.heads, a.dim, a.vdim = rows.rows, rows.segments, heads, dim, vdim
    a.q, a.k, a.v, a.stride = q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0)
    a.decay_pow, a.state, a.num_slots, a.out, a.dtype = _ptr(powers), state.data_ptr(), int(state.shape[0]), out.data_ptr(), dtype_code(q.dtype)
    a.slot_stride, a.q_scale, a.key_heads, a.skip = state.stride(0), float(q_scale), 0 if key_heads is None else key_heads, _ptr(skip)
    if gated is not None:
        a.log_decay, a.log_take, a.normaliser = (_ptr(t) for t in gated)
    return a


def recurrence_simple(a: RecurrenceArgs) -> None:
    check(_lib.load_group("recurrence").cacheir_b200_recurrence_simple(ctypes.byref(a), _stream()), "recurrence_simple")


def recurrence_step(a: RecurrenceArgs) -> None:
    check(_lib.load_group("recurrence").cacheir_b200_recurrence_step(ctypes.byref(a), _stream()), "recurrence_step")


def recurrence_chunked_supported(dim: int, vdim: int, dtype: torch.dtype) -> bool:
    return bool(_lib.load_group("recurrence").cacheir_b200_recurrence_chunked_supported(dim, vdim, dtype_code(dtype)))


def recurrence_workspace_bytes(rows: int, segments: int, heads: int, dim: int, vdim: int) -> int:
    return int(_lib.load_group("recurrence").cacheir_b200_recurrence_workspace_bytes(rows, segments, heads, dim, vdim))


def recurrence_chunked(a: RecurrenceArgs, workspace: torch.Tensor | None) -> None:
    check(_lib.load_group("recurrence").cacheir_b200_recurrence_chunked(
        ctypes.byref(a), _ptr(workspace), 0 if workspace is None else workspace.numel() * workspace.element_size(), _stream()),
        "recurrence_chunked")


# ---- matrix memory -------------------------------------------------------------------------------------------------------
def memory_state_size(heads: int, dim: int, vdim: int) -> int:
    """float32 entries of one sequence's state: matrices, normalisers, running maxima; whole 16-byte pieces."""
    return (heads * (dim * vdim + dim + 1) + 3) // 4 * 4


@dataclass
class MemoryGates:
    """Gate logits [T, 2*heads] float32 (input gates, then forget gates), their biases [heads] and the cap."""

    logits: torch.Tensor
    in_bias: torch.Tensor
    forget_bias: torch.Tensor
    cap: float

    def args(self) -> tuple:
        _require_cuda(self.logits, self.in_bias, self.forget_bias)
        _f32(self.in_bias, self.forget_bias)
        if self.logits.dtype != torch.float32 or self.logits.stride(1) != 1 or int(self.logits.shape[1]) != 2 * self.in_bias.numel():
            raise ValueError("gate logits are float32 [T, 2*heads] with dense rows")
        return (self.logits.data_ptr(), self.logits.stride(0), self.in_bias.data_ptr(), self.forget_bias.data_ptr(), float(self.cap))


def memory_gates(a: RecurrenceArgs, gates: MemoryGates, log_decay: torch.Tensor, log_take: torch.Tensor, maximum: torch.Tensor) -> None:
    _require_cuda(log_decay, log_take, maximum)
    check(_lib.load_group("recurrence").cacheir_b200_memory_gates(
        ctypes.byref(a), *gates.args(), log_decay.data_ptr(), log_take.data_ptr(), maximum.data_ptr(), _stream()), "memory_gates")


def _memory_gate(gate: torch.Tensor, weight: torch.Tensor, columns: int) -> None:
    _require_cuda(gate, weight)
    _f32(weight)
    if gate.stride(1) != 1 or int(gate.shape[1]) != columns or weight.numel() != columns:
        raise ValueError("the output gate and the norm weight have one column per output column")


def memory_norm(o: torch.Tensor, normaliser: torch.Tensor, maximum: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, eps: float,
                out: torch.Tensor, *, heads: int, vdim: int) -> torch.Tensor:
    _require_cuda(o, normaliser, maximum, out)
    _f32(normaliser, maximum)
    _memory_gate(gate, weight, heads * vdim)
    if not o.is_contiguous() or not out.is_contiguous() or o.shape != out.shape or int(o.shape[1]) != heads * vdim:
        raise ValueError("memory_norm expects contiguous [T, heads*vdim] o and out")
    check(_lib.load_group("recurrence").cacheir_b200_memory_norm(
        o.data_ptr(), normaliser.data_ptr(), maximum.data_ptr(), gate.data_ptr(), gate.stride(0), weight.data_ptr(), float(eps), out.data_ptr(),
        int(o.shape[0]), heads, vdim, dtype_code(o.dtype), _stream()), "memory_norm")
    return out


def memory_step(a: RecurrenceArgs, gates: MemoryGates, gate: torch.Tensor, weight: torch.Tensor, eps: float) -> None:
    _memory_gate(gate, weight, a.heads * a.vdim)
    check(_lib.load_group("recurrence").cacheir_b200_memory_step(
        ctypes.byref(a), *gates.args(), gate.data_ptr(), gate.stride(0), weight.data_ptr(), float(eps), _stream()), "memory_step")


# ---- state space -----------------------------------------------------------------------------------------------------------
@dataclass
class StepSizes:
    """Step size logits [T, heads] float32 (a view with dense rows), their bias and the logarithm of the decay rate [heads]."""

    logits: torch.Tensor
    bias: torch.Tensor
    log_rate: torch.Tensor

    def args(self) -> tuple:
        _require_cuda(self.logits, self.bias, self.log_rate)
        _f32(self.bias, self.log_rate)
        if self.logits.dtype != torch.float32 or self.logits.stride(1) != 1 or not int(self.logits.shape[1]) == self.bias.numel() == self.log_rate.numel():
            raise ValueError("step size logits are float32 [T, heads] with dense rows")
        return (self.logits.data_ptr(), self.logits.stride(0), self.bias.data_ptr(), self.log_rate.data_ptr())


def state_space_gates(a: RecurrenceArgs, steps: StepSizes, log_decay: torch.Tensor, log_take: torch.Tensor) -> None:
    _require_cuda(log_decay, log_take)
    check(_lib.load_group("recurrence").cacheir_b200_state_space_gates(
        ctypes.byref(a), *steps.args(), log_decay.data_ptr(), log_take.data_ptr(), _stream()), "state_space_gates")


def state_space_step(a: RecurrenceArgs, steps: StepSizes) -> None:
    check(_lib.load_group("recurrence").cacheir_b200_state_space_step(ctypes.byref(a), *steps.args(), _stream()), "state_space_step")


def device_status(reset: bool = True) -> int:
    return _lib.group_device_status(reset)
