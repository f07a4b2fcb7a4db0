"""Torch-tensor wrappers over include/cacheir_b200_talking.h and cacheir_b200_delta.h: talking-heads attention, short
convolutions, the gated delta rule. Same rules as `hybrid_ops`."""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from ._lib import ConvArgs, DeltaArgs, TalkingArgs, check
from .hybrid_ops import Rows, _f32
from .ops import _ptr, _require_cuda, _stream, dtype_code


# ---- talking-heads attention -------------------------------------------------------------------------------------------------
def talking_args(rows: Rows, keys: torch.Tensor, values: torch.Tensor, talk: torch.Tensor, *, heads: int, kv_heads: int, dim: int, vdim: int,
                 window: int, scale: float) -> TalkingArgs:
    """keys [slots, page, kv_heads*dim], values [slots, page, kv_heads*vdim], talk [heads, heads] float32."""
    _require_cuda(keys, values, talk)
    _f32(talk)
    for pool, d in ((keys, dim), (values, vdim)):
        if pool.dim() != 3 or int(pool.shape[2]) != kv_heads * d or not pool.is_contiguous():
            raise ValueError(f"a pool must be a contiguous [slots, page, {kv_heads * d}] tensor")
    if keys.shape[:2] != values.shape[:2] or keys.dtype != values.dtype or tuple(talk.shape) != (heads, heads) or heads % kv_heads:
        raise ValueError("keys and values have the same rows and type, talk one entry per pair of heads")
    a = TalkingArgs()
    a.positions, a.row_seg, a.cu_rows = rows.positions.data_ptr(), rows.row_seg.data_ptr(), rows.cu_rows.data_ptr()
    a.page_table, a.rows, a.segments = rows.page_table.data_ptr(), rows.rows, rows.segments
    a.max_pages, a.page_size, a.num_slots = int(rows.page_table.shape[1]), int(keys.shape[1]), int(keys.shape[0])
    a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale = heads, kv_heads, dim, vdim, window, float(scale)
    a.talk, a.keys, a.values, a.dtype, a.decode = talk.data_ptr(), keys.data_ptr(), values.data_ptr(), dtype_code(keys.dtype), int(rows.decode)
    return a


def talking_prepare(a: TalkingArgs, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, q_out: torch.Tensor, *, eps: float,
                    table: torch.Tensor | None, mixed: bool) -> None:
    """Cache rows of k and v; rotated queries [T, heads*dim], or `mixed` ones [T, heads*kv_heads*dim], in `q_out`."""
    _require_cuda(q, k, v, q_out, table)
    sizes = (a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim)
    if any(t.stride(1) != 1 or int(t.shape[1]) != n for t, n in zip((q, k, v), sizes)):
        raise ValueError("q, k and v have the columns of their heads and dense rows")
    if not q_out.is_contiguous() or int(q_out.shape[1]) != sizes[0] * (a.kv_heads if mixed else 1):
        raise ValueError("q_out is a contiguous [T, heads*dim] tensor, times kv_heads columns for mixed queries")
    check(_lib.load_group("talking").cacheir_b200_talking_prepare(
        ctypes.byref(a), q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0),
        0 if table is None else 2 * int(table.shape[1]), _ptr(table), (1 << 30) if table is None else int(table.shape[0]), float(eps), int(mixed),
        q_out.data_ptr(), _stream()), "talking_prepare")


def _talk(a: TalkingArgs, q: torch.Tensor, out: torch.Tensor, mixed: bool) -> tuple:
    _require_cuda(q, out)
    if not q.is_contiguous() or not out.is_contiguous() or int(out.shape[1]) != a.heads * a.vdim or int(q.shape[1]) != a.heads * a.dim * (a.kv_heads if mixed else 1):
        raise ValueError("talking attention expects contiguous prepared queries and a [T, heads*vdim] out")
    return (ctypes.byref(a), q.data_ptr(), out.data_ptr())


def talking_simple(a: TalkingArgs, q: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    check(_lib.load_group("talking").cacheir_b200_talking_simple(*_talk(a, q, out, False), _stream()), "talking_simple")
    return out


def talking_step_supported(heads: int, kv_heads: int, dim: int, vdim: int, page_size: int, dtype: torch.dtype) -> bool:
    return bool(_lib.load_group("talking").cacheir_b200_talking_step_supported(heads, kv_heads, dim, vdim, page_size, dtype_code(dtype)))


def talking_step_splits(rows: int, heads: int, kv_heads: int, dim: int, vdim: int, window: int, max_pages: int, page_size: int) -> int:
    return int(_lib.load_group("talking").cacheir_b200_talking_step_splits(rows, heads, kv_heads, dim, vdim, window, max_pages, page_size))


def talking_step(a: TalkingArgs, q: torch.Tensor, out: torch.Tensor, *, splits: int = 0) -> torch.Tensor:
    check(_lib.load_group("talking").cacheir_b200_talking_step(*_talk(a, q, out, False), int(splits), _stream()), "talking_step")
    return out


def talking_prompt_supported(heads: int, kv_heads: int, dim: int, vdim: int, page_size: int, dtype: torch.dtype) -> bool:
    return bool(_lib.load_group("talking").cacheir_b200_talking_prompt_supported(heads, kv_heads, dim, vdim, page_size, dtype_code(dtype)))


def talking_prompt(a: TalkingArgs, q: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    check(_lib.load_group("talking").cacheir_b200_talking_prompt(*_talk(a, q, out, True), _stream()), "talking_prompt")
    return out


# ---- short convolution ---------------------------------------------------------------------------------------------------------
def short_conv(rows: Rows, x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor | None, state: torch.Tensor, offset: int,
               out: torch.Tensor) -> torch.Tensor:
    """out = silu(causal convolution of x [T, channels]); weight [channels, taps] float32. The last taps - 1 inputs of a sequence lie
    in its state slot (state [slots, size] float32) from `offset` on."""
    _require_cuda(x, weight, bias, state, out)
    _f32(weight, state, *([] if bias is None else [bias]))
    channels, taps = (int(n) for n in weight.shape)
    if int(x.shape[1]) != channels or x.stride(1) != 1 or out.stride(1) != 1 or int(out.shape[1]) != channels or out.dtype != x.dtype:
        raise ValueError("x and out have a column per channel, dense rows and one type")
    if state.dim() != 2 or int(state.shape[1]) < offset + (taps - 1) * channels or (bias is not None and bias.numel() != channels):
        raise ValueError("a state slot must hold the last taps - 1 inputs, bias have an entry per channel")
    a = ConvArgs()
    a.positions, a.cu_rows, a.slots = rows.positions.data_ptr(), rows.cu_rows.data_ptr(), rows.slots.data_ptr()
    a.rows, a.segments, a.channels, a.taps = rows.rows, rows.segments, channels, taps
    a.x, a.stride, a.w, a.bias = x.data_ptr(), x.stride(0), weight.data_ptr(), _ptr(bias)
    a.state, a.slot_stride, a.num_slots, a.dtype = state.data_ptr() + 4 * offset, state.stride(0), int(state.shape[0]), dtype_code(x.dtype)
    a.out, a.out_stride = out.data_ptr(), out.stride(0)
    check(_lib.load_group("delta").cacheir_b200_short_conv(ctypes.byref(a), _stream()), "short_conv")
    return out


# ---- gated delta rule ------------------------------------------------------------------------------------------------------------
def delta_args(rows: Rows, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, logits: torch.Tensor, bias: torch.Tensor, log_rate: torch.Tensor,
               state: torch.Tensor, out: torch.Tensor, *, heads: int, key_heads: int, dim: int, vdim: int) -> DeltaArgs:
    """q, k [T, key_heads*dim] and v [T, heads*vdim] with one row stride, logits [T, 2*heads] float32 (beta, then decay), bias and
    log_rate [heads]; state rows begin with [heads, dim, vdim]."""
    _require_cuda(q, k, v, logits, bias, log_rate, state, out)
    _f32(bias, log_rate, state)
    if not (q.stride(0) == k.stride(0) == v.stride(0)) or q.stride(1) != 1 or k.stride(1) != 1 or v.stride(1) != 1:
        raise ValueError("q, k and v must share one row stride and have dense rows")
    if int(q.shape[1]) != key_heads * dim or int(k.shape[1]) != key_heads * dim or int(v.shape[1]) != heads * vdim or heads % key_heads:
        raise ValueError("q, k and v have the columns of their heads")
    if logits.dtype != torch.float32 or logits.stride(1) != 1 or int(logits.shape[1]) != 2 * heads or bias.numel() != heads or log_rate.numel() != heads:
        raise ValueError("logits are float32 [T, 2*heads] with dense rows, bias and log_rate [heads]")
    if not out.is_contiguous() or int(out.shape[1]) != heads * vdim or state.stride(0) < heads * dim * vdim:
        raise ValueError("out is a contiguous [T, heads*vdim] tensor, a state slot holds [heads, dim, vdim]")
    a = DeltaArgs()
    a.positions, a.cu_rows, a.slots = rows.positions.data_ptr(), rows.cu_rows.data_ptr(), rows.slots.data_ptr()
    a.rows, a.segments, a.heads, a.key_heads, a.dim, a.vdim = rows.rows, rows.segments, heads, key_heads, dim, vdim
    a.q, a.k, a.v, a.stride, a.z, a.z_stride = q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), logits.data_ptr(), logits.stride(0)
    a.bias, a.log_rate, a.state, a.slot_stride = bias.data_ptr(), log_rate.data_ptr(), state.data_ptr(), state.stride(0)
    a.num_slots, a.dtype, a.out = int(state.shape[0]), dtype_code(q.dtype), out.data_ptr()
    return a


def delta_simple(a: DeltaArgs) -> None:
    check(_lib.load_group("delta").cacheir_b200_delta_simple(ctypes.byref(a), _stream()), "delta_simple")


def delta_step(a: DeltaArgs, gate: torch.Tensor, weight: torch.Tensor, eps: float) -> None:
    """One token per sequence, with the head's norm (weight [vdim]) and the silu gate behind it."""
    _require_cuda(gate, weight)
    _f32(weight)
    if gate.stride(1) != 1 or int(gate.shape[1]) != a.heads * a.vdim or weight.numel() != a.vdim:
        raise ValueError("the gate has one column per output column, the weight one entry per column of a head")
    check(_lib.load_group("delta").cacheir_b200_delta_step(ctypes.byref(a), gate.data_ptr(), gate.stride(0), weight.data_ptr(), float(eps), _stream()),
          "delta_step")


def delta_chunked_supported(dim: int, vdim: int, dtype: torch.dtype) -> bool:
    return bool(_lib.load_group("delta").cacheir_b200_delta_chunked_supported(dim, vdim, dtype_code(dtype)))


def delta_workspace_bytes(rows: int, segments: int, heads: int) -> int:
    return int(_lib.load_group("delta").cacheir_b200_delta_workspace_bytes(rows, segments, heads))


def delta_chunked(a: DeltaArgs, workspace: torch.Tensor) -> None:
    check(_lib.load_group("delta").cacheir_b200_delta_chunked(ctypes.byref(a), workspace.data_ptr(), workspace.numel() * workspace.element_size(),
                                                             _stream()), "delta_chunked")
