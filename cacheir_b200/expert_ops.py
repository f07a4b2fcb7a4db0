"""Torch-tensor wrappers over include/cacheir_b200_experts.h: tied attention and mixtures of experts. Same rules as
`hybrid_ops`."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from ._lib import DenseArgs, RouteRule, TiedArgs, check
from .hybrid_ops import DENSE_CLAMPED_GLU, DENSE_PLAIN, DENSE_SWIGLU, NEXT_COPY, NEXT_NONE, Next, Rows, _f32, _next
from .ops import _ptr, _require_cuda, _stream, dtype_code


# ---- tied attention --------------------------------------------------------------------------------------------------
def row_layout(dim: int, rot_dims: int, key_dim: int | None = None) -> tuple[int, int]:
    """(width, first key column) of a cached row with `dim` value columns: values that are the keys, or (`key_dim`) keys of
    their own behind them."""
    return (dim + rot_dims, rot_dims) if key_dim is None else (dim + key_dim, dim)


def query_width(dim: int, rot_dims: int, key_dim: int | None = None) -> int:
    """Columns of a prepared query: a cached row without the whole 64-column boxes that would meet zeros."""
    width, key_from = row_layout(dim, rot_dims, key_dim)
    return width - key_from // 64 * 64


def tied_args(rows: Rows, pool: torch.Tensor, inv_rms: torch.Tensor, *, heads: int, kv_heads: int, dim: int, rot_dims: int, window: int,
              keep_first: int, scale: float, softcap: float | None, sink: torch.Tensor | None, key_dim: int | None = None,
              reach: float | None = None) -> TiedArgs:
    """pool [slots, kv_heads, page, width] (see row_layout), inv_rms [slots, kv_heads, page] float32. `reach`: what |q . key|
    never exceeds, 0 if no bound is known; by default that of unit root mean squares."""
    _require_cuda(pool, inv_rms, sink)
    width, key_from = row_layout(dim, rot_dims, key_dim)
    if pool.dim() != 4 or int(pool.shape[1]) != kv_heads or int(pool.shape[3]) != width or not pool.is_contiguous():
        raise ValueError(f"the pool must be a contiguous [slots, kv_heads, page, {width}] tensor")
    _f32(inv_rms, *([] if sink is None else [sink]))
    if inv_rms.shape != pool.shape[:3] or (sink is not None and sink.numel() != heads):
        raise ValueError("inv_rms has one entry per cached row, sink one per head")
    a = TiedArgs()
    a.positions, a.row_seg, a.cu_rows = rows.positions.data_ptr(), rows.row_seg.data_ptr(), rows.cu_rows.data_ptr()
    a.page_table, a.rows, a.segments = rows.page_table.data_ptr(), rows.rows, rows.segments
    a.max_pages, a.page_size, a.num_slots = int(rows.page_table.shape[1]), int(pool.shape[2]), int(pool.shape[0])
    a.heads, a.kv_heads, a.dim, a.width, a.key_from, a.window, a.keep_first = heads, kv_heads, dim, width, key_from, window, keep_first
    a.scale, a.cap = float(scale), 0.0 if softcap is None else float(softcap)
    a.reach = float(dim if key_dim is None else key_dim) if reach is None else float(reach)
    a.pool, a.inv_rms, a.sink = pool.data_ptr(), inv_rms.data_ptr(), _ptr(sink)
    a.dtype, a.decode = dtype_code(pool.dtype), int(rows.decode)
    return a


def tied_prepare(a: TiedArgs, q: torch.Tensor, k: torch.Tensor, q_out: torch.Tensor, *, eps: float, table: torch.Tensor | None,
                 v: torch.Tensor | None = None, q_weight: torch.Tensor | None = None, k_weight: torch.Tensor | None = None,
                 whole: bool = False) -> None:
    """Cache rows of `k` [T, kv_heads*d] (and `v` [T, kv_heads*dim], if the values are not the keys); prepared queries of `q`
    [T, heads*d] in `q_out`. Weights have an entry per column of a head, or with `whole` (one norm over all heads) of the
    projection."""
    _require_cuda(q, k, v, q_out, table, q_weight, k_weight)
    d = a.dim if v is None else a.width - a.dim
    if q.stride(1) != 1 or k.stride(1) != 1 or not q_out.is_contiguous() or int(q_out.shape[1]) != a.heads * (a.width - a.key_from // 64 * 64):
        raise ValueError("tied_prepare expects dense rows and a contiguous [T, heads * query_width] output")
    if int(q.shape[1]) != a.heads * d or int(k.shape[1]) != a.kv_heads * d or (v is not None and (v.stride(1) != 1 or int(v.shape[1]) != a.kv_heads * a.dim)):
        raise ValueError("q, k and v have the columns of their heads")
    for w, heads in ((q_weight, a.heads), (k_weight, a.kv_heads)):
        if w is not None:
            _f32(w)
            if w.numel() != (heads * d if whole else d):
                raise ValueError("norm weights have an entry per column of what they normalise")
    check(_lib.load_group("experts").cacheir_b200_tied_prepare(
        ctypes.byref(a), q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), _ptr(v), 0 if v is None else v.stride(0),
        0 if table is None else 2 * int(table.shape[1]), int(whole), _ptr(q_weight), _ptr(k_weight), float(eps), _ptr(table),
        (1 << 30) if table is None else int(table.shape[0]), q_out.data_ptr(), _stream()), "tied_prepare")


def _attend(a: TiedArgs, q: torch.Tensor, gate: torch.Tensor | None, out: torch.Tensor) -> tuple:
    _require_cuda(q, gate, out)
    if not q.is_contiguous() or not out.is_contiguous() or int(out.shape[1]) != a.heads * a.dim:
        raise ValueError("tied attention expects contiguous q and [T, heads*dim] out")
    if gate is not None and (gate.stride(1) != 1 or int(gate.shape[1]) != a.heads * a.dim):
        raise ValueError("the gate has one column per output column")
    return (ctypes.byref(a), q.data_ptr(), _ptr(gate), 0 if gate is None else gate.stride(0), out.data_ptr())


def tied_attention_simple(a: TiedArgs, q: torch.Tensor, gate: torch.Tensor | None, out: torch.Tensor) -> torch.Tensor:
    check(_lib.load_group("experts").cacheir_b200_tied_attention_simple(*_attend(a, q, gate, out), _stream()), "tied_attention_simple")
    return out


def tied_prompt_supported(heads: int, kv_heads: int, dim: int, rot_dims: int, page_size: int, dtype: torch.dtype,
                          key_dim: int | None = None) -> bool:
    return bool(_lib.load_group("experts").cacheir_b200_tied_prompt_supported(heads, kv_heads, dim, *row_layout(dim, rot_dims, key_dim), page_size,
                                                                              dtype_code(dtype)))


def tied_attention_prompt(a: TiedArgs, q: torch.Tensor, gate: torch.Tensor | None, out: torch.Tensor) -> torch.Tensor:
    check(_lib.load_group("experts").cacheir_b200_tied_attention_prompt(*_attend(a, q, gate, out), _stream()), "tied_attention_prompt")
    return out


def tied_step_supported(heads: int, kv_heads: int, dim: int, rot_dims: int, page_size: int, dtype: torch.dtype,
                        key_dim: int | None = None) -> bool:
    return bool(_lib.load_group("experts").cacheir_b200_tied_step_supported(heads, kv_heads, dim, *row_layout(dim, rot_dims, key_dim), page_size,
                                                                            dtype_code(dtype)))


def tied_step_splits(rows: int, heads: int, kv_heads: int, window: int, keep_first: int, max_pages: int, page_size: int) -> int:
    return int(_lib.load_group("experts").cacheir_b200_tied_step_splits(rows, heads, kv_heads, window, keep_first, max_pages, page_size))


def tied_attention_step(a: TiedArgs, q: torch.Tensor, gate: torch.Tensor | None, out: torch.Tensor, *, splits: int = 0) -> torch.Tensor:
    check(_lib.load_group("experts").cacheir_b200_tied_attention_step(*_attend(a, q, gate, out), int(splits), _stream()), "tied_attention_step")
    return out


# ---- mixtures of experts -----------------------------------------------------------------------------------------------
@dataclass
class Routing:
    """Which rows go where: places in expert order (see the header)."""

    experts: int
    top: int
    counters: torch.Tensor       # [experts + 1] zeros
    cu: torch.Tensor             # [experts + 1]
    token_of: torch.Tensor       # [rows * top]
    place_of: torch.Tensor       # [rows, top]
    chosen: torch.Tensor         # [rows, top]
    weight: torch.Tensor         # [rows, top] float32

    @property
    def places(self) -> int:
        return int(self.token_of.numel())


@dataclass
class SoftmaxRule:
    """Choices by softmax + correction within the `keep` best of `groups` groups of neighbours; the last `identity` logits
    stand for the token itself."""

    correction: torch.Tensor | None = None
    groups: int = 1
    keep: int = 1
    identity: int = 0


def route(logits: torch.Tensor, row_seg: torch.Tensor, routing: Routing, scale: float, x: torch.Tensor | None = None,
          placed: torch.Tensor | None = None, rule: SoftmaxRule | None = None) -> None:
    """Choices and places; with `placed` [rows * top, width] also a copy of every row of `x` at its places. Without a rule
    choices go by the logits and weights are their sigmoids."""
    _require_cuda(logits, row_seg, routing.counters)
    rows = int(logits.shape[0])
    if logits.dtype != torch.float32 or logits.stride(1) != 1 or tuple(routing.place_of.shape) != (rows, routing.top):
        raise ValueError("route takes float32 logits with dense rows and a routing of their row count")
    if placed is not None and (x is None or not x.is_contiguous() or not placed.is_contiguous() or x.dtype != placed.dtype
                               or int(x.shape[0]) != rows or tuple(placed.shape) != (routing.places, int(x.shape[1]))):
        raise ValueError("placed has a row per place, x one per logits row, both dense")
    r = RouteRule(groups=1, keep=1, scale=float(scale))
    if rule is not None:
        r.softmax, r.identity, r.groups, r.keep = 1, rule.identity, rule.groups, rule.keep
        if rule.correction is not None:
            _require_cuda(rule.correction)
            _f32(rule.correction)
            r.correction = rule.correction.data_ptr()
    scored = routing.experts + r.identity
    if int(logits.shape[1]) < scored or (r.correction and rule.correction.numel() != scored):
        raise ValueError("logits and correction have a column per expert and identity expert")
    check(_lib.load_group("experts").cacheir_b200_route(
        logits.data_ptr(), logits.stride(0), row_seg.data_ptr(), rows, routing.experts, routing.top, ctypes.byref(r), routing.counters.data_ptr(),
        routing.cu.data_ptr(), routing.token_of.data_ptr(), routing.place_of.data_ptr(), routing.weight.data_ptr(),
        routing.chosen.data_ptr(), None if placed is None else x.data_ptr(), _ptr(placed),
        0 if placed is None else int(x.shape[1]) * x.element_size(), _stream()), "route")


def grouped_supported(k: int, x_stride: int, dtype: torch.dtype) -> bool:
    return dtype == torch.bfloat16 and k % 8 == 0 and x_stride % 8 == 0


def grouped_all_rows() -> int:
    """Rows of a step up to which an expert multiplies all of them and keeps those that chose it."""
    return int(_lib.load_group("experts").cacheir_b200_grouped_all_rows())


def grouped_gemm(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, routing: Routing, *, by_row: bool, epilogue: int = DENSE_PLAIN,
                 limit: float = 0.0) -> torch.Tensor:
    """out[place] = f(x[.] W_e^T), w [experts*N, K]; x has a row per token (`by_row`, see grouped_all_rows) or per place."""
    _require_cuda(x, w, out)
    n = int(w.shape[0]) // routing.experts
    cols = n // 2 if epilogue in (DENSE_SWIGLU, DENSE_CLAMPED_GLU) else n
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or x.stride(1) != 1 or w.stride(1) != 1 or out.dtype != torch.bfloat16:
        raise ValueError("grouped_gemm takes bf16 operands with dense rows")
    if int(out.shape[0]) != routing.places or int(out.shape[1]) < cols or out.stride(1) != 1 or int(x.shape[0]) != (routing.places // routing.top if by_row else routing.places):
        raise ValueError("out must have a row per place, x one per place or token")
    a = DenseArgs()
    a.x, a.w, a.y, a.T, a.N, a.K, a.batch, a.w_batch_rows = x.data_ptr(), w.data_ptr(), out.data_ptr(), routing.places, n, int(w.shape[1]), routing.experts, n
    a.epilogue, a.w_stride, a.x_stride, a.y_stride, a.limit = epilogue, w.stride(0), x.stride(0), out.stride(0), float(limit)
    check(_lib.load_group("experts").cacheir_b200_grouped_gemm(
        ctypes.byref(a), routing.cu.data_ptr(), routing.place_of.data_ptr() if by_row else None, routing.top, int(x.shape[0]), _stream()), "grouped_gemm")
    return out


def grouped_simple(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, routing: Routing, *, gather: bool) -> torch.Tensor:
    """The plain grouped product in float32 arithmetic, any extents."""
    _require_cuda(x, w, out)
    n = int(w.shape[0]) // routing.experts
    if x.dtype != w.dtype or out.dtype != x.dtype or x.stride(1) != 1 or w.stride(1) != 1 or out.stride(1) != 1 or int(out.shape[0]) != routing.places:
        raise ValueError("grouped_simple takes operands of one type with dense rows and an out row per place")
    check(_lib.load_group("experts").cacheir_b200_grouped_simple(
        x.data_ptr(), w.data_ptr(), out.data_ptr(), routing.cu.data_ptr(), routing.token_of.data_ptr() if gather else None, routing.places,
        routing.experts, n, int(w.shape[1]), w.stride(0), x.stride(0), out.stride(0), dtype_code(x.dtype), _stream()), "grouped_simple")
    return out


def combine_residual_rms(residual: torch.Tensor, y: torch.Tensor, routing: Routing, shared: torch.Tensor | None, weight: torch.Tensor,
                         eps: float, nx: Next | None = None) -> None:
    """residual += rms_norm(sum of the chosen experts' rows by weight + shared) * weight"""
    _require_cuda(residual, y, shared, weight)
    _f32(residual, weight)
    if not y.is_contiguous() or y.shape[1] != residual.shape[1] or (shared is not None and (shared.shape != residual.shape or not shared.is_contiguous())):
        raise ValueError("y and shared have the residual's width and dense rows")
    if nx is not None and (nx.norm is not None or nx.out.shape != residual.shape or not nx.out.is_contiguous()):
        raise ValueError("the combine leaves a copy of the residual or nothing")
    check(_lib.load_group("experts").cacheir_b200_combine_residual_rms(
        residual.data_ptr(), y.data_ptr(), routing.place_of.data_ptr(), routing.weight.data_ptr(), routing.top, _ptr(shared), weight.data_ptr(),
        float(eps), int(residual.shape[0]), int(residual.shape[1]), NEXT_NONE if nx is None else NEXT_COPY,
        None if nx is None else nx.out.data_ptr(), dtype_code(y.dtype), _stream()), "combine_residual_rms")


def combine_residual(residual: torch.Tensor, y: torch.Tensor, routing: Routing, x: torch.Tensor, shared: torch.Tensor | None,
                     shared_gate: torch.Tensor | None, nx: Next | None = None) -> None:
    """residual += sum of the chosen experts' rows (or x's own, for identity experts) by weight + shared * sigmoid(shared_gate);
    shared_gate is a column [rows] of a float32 tensor. `nx.out` may be `x`."""
    _require_cuda(residual, y, x, shared, shared_gate)
    _f32(residual)
    if any(t is not None and (t.shape != residual.shape or not t.is_contiguous() or t.dtype != y.dtype) for t in (x, shared)):
        raise ValueError("x and shared have the residual's shape and y's type")
    if not y.is_contiguous() or y.shape[1] != residual.shape[1] or (nx is not None and (nx.out.shape != residual.shape or not nx.out.is_contiguous())):
        raise ValueError("y and the next operator's input have the residual's width and dense rows")
    if shared_gate is not None and (shared_gate.dtype != torch.float32 or shared_gate.dim() != 1 or shared_gate.numel() != residual.shape[0]):
        raise ValueError("shared_gate is one float32 entry per row")
    check(_lib.load_group("experts").cacheir_b200_combine_residual(
        residual.data_ptr(), y.data_ptr(), routing.place_of.data_ptr(), routing.weight.data_ptr(), routing.top, x.data_ptr(), _ptr(shared),
        _ptr(shared_gate), 0 if shared_gate is None else shared_gate.stride(0), int(residual.shape[0]), int(residual.shape[1]), *_next(nx),
        dtype_code(y.dtype), _stream()), "combine_residual")
