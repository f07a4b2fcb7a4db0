"""Ragged steps: portions of prompts beside single decoded tokens as one pass through a lowered graph.

`RaggedPlan` is the plan class of families whose layers need to know which rows belong to one sequence (linear
recurrences, windowed attention over tiles of neighbouring tokens) or which rows are real (mixtures of experts). It keeps `_DecodePlan`'s contract (static buffers,
a flat launch list, CUDA-graph replay from the second step) and adds the segment arrays. A decode plan has one row per
sequence and advances on the device; a portion plan has room for `rows` rows of `segments` sequences and takes its
metadata in one copy per step. Residual stream float32; in bfloat16 runs each sublayer boundary (norm, residual add,
next norm) is the epilogue of the GEMM in front of it.
"""
from __future__ import annotations

from typing import Any, Callable

import numpy as np
import torch

from . import expert_ops as X
from . import hybrid_ops as H
from . import mixer_ops as M
from . import ops

# rows a portion plan is made for: one plan (and one CUDA graph) per bucket, not per portion length
ROW_BUCKETS = (1, 2, 4, 8, 16, 32, 64, 128, 192, 256, 384, 512, 768, 1024, 1536, 2048, 3072, 4096)


def bucket(n: int) -> int:
    for b in ROW_BUCKETS:
        if n <= b:
            return b
    return (n + 1023) // 1024 * 1024


GLU_LABELS = {"gelu_tanh": ".geglu", "silu": ".swiglu", "clamped": ".clamped_glu"}
# ops that take the residual stream itself, as a copy in the activation type
READS_RESIDUAL = {"token_side_gate", "concat_matmul", "fused_glu", "expert_router"}


def rotary_frequencies(dims: int, base: float, scaling: tuple[float, float, float, float] | None = None) -> np.ndarray:
    """base^(-2i/dims) in double precision. `scaling` = (factor, low, high, original): wavelengths above original/low are
    stretched by factor, those below original/high kept, and the blend between is linear in original/wavelength."""
    freq = float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    if scaling is None:
        return freq
    factor, low, high, original = scaling
    turns = original * freq / (2.0 * np.pi)              # original / wavelength
    with np.errstate(divide="ignore", invalid="ignore"):
        keep = (turns - low) / (high - low)
    blended = (1.0 - keep) * freq / factor + keep * freq
    return np.where(turns > high, freq, np.where(turns < low, freq / factor, blended))


def rotate_half_table(positions: int, dims: int, base: float, scaling: tuple[float, float, float, float] | None = None) -> np.ndarray:
    """float32 [positions, dims/2, 2] (cos, sin) of position times frequency, evaluated in double precision."""
    freq = rotary_frequencies(dims, base, scaling)
    angle = np.arange(positions, dtype=np.float64)[:, None] * freq[None, :]
    return np.stack([np.cos(angle), np.sin(angle)], axis=-1).astype(np.float32)


def yarn_frequencies(dims: int, base: float, factor: float, original: float, fast: float, slow: float) -> tuple[np.ndarray, float]:
    """(frequencies in double precision, factor of cosine and sine): pairs that turn more than `fast` times within `original`
    positions keep their frequency, those that turn less than `slow` times have it divided by `factor`, with a linear ramp over the
    pairs between."""
    freq = rotary_frequencies(dims, base)

    def pair(turns: float) -> float:
        return dims * np.log(original / (2.0 * np.pi * turns)) / (2.0 * np.log(base))
    lo, hi = max(np.floor(pair(fast)), 0.0), min(np.ceil(pair(slow)), dims - 1.0)
    ramp = np.clip((np.arange(dims // 2, dtype=np.float64) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * float(np.log(factor)) + 1.0


def yarn_table(positions: int, dims: int, base: float, yarn: tuple[float, float, float, float]) -> np.ndarray:
    """`rotate_half_table` of `yarn_frequencies`, cosine and sine with their factor."""
    freq, factor = yarn_frequencies(dims, base, *yarn)
    angle = np.arange(positions, dtype=np.float64)[:, None] * freq[None, :]
    return (np.stack([np.cos(angle), np.sin(angle)], axis=-1) * factor).astype(np.float32)


def make_plan_class(base: type) -> type:
    """`RaggedPlan` over the runtime's plan class (the runtime module imports this one)."""

    class RaggedPlan(base):
        def __init__(self, engine: Any, rows: int, width: int, *, segments: int | None = None, logit_rows: int | None = None):
            self.engine = engine
            self.decode = segments is None
            self.batch = rows
            self.segments = rows if segments is None else segments
            self.width = width
            self.logit_rows = rows if logit_rows is None else logit_rows
            self.pool_generation = engine.allocator.generation
            dev = engine.device
            # int32 metadata in one block, so that a portion step needs one copy
            parts = {"lens": rows, "row_seg": rows, "cu_rows": self.segments + 1, "slots": self.segments, "logit_index": self.logit_rows,
                     "table": self.segments * width}
            offsets = np.cumsum([0] + [(n + 3) // 4 * 4 for n in parts.values()])
            self._host_meta = torch.zeros((int(offsets[-1]),), dtype=torch.int32).pin_memory()
            self._meta = torch.zeros((int(offsets[-1]),), device=dev, dtype=torch.int32)
            device, host = {}, {}
            for (name, n), off in zip(parts.items(), offsets):
                device[name], host[name] = self._meta[off:off + n], self._host_meta[off:off + n]
            self.seq_lens, self.host_lens = device["lens"], host["lens"]
            self.page_table, self.host_table = device["table"].view(self.segments, width), host["table"].view(self.segments, width)
            self._host = host
            self._device_slots = device["slots"]
            self.logit_index = None if self.decode else device["logit_index"]
            self.ids = torch.zeros((rows,), device=dev, dtype=torch.int64)
            self.host_ids = torch.zeros((rows,), dtype=torch.int64).pin_memory()
            self.positions = torch.zeros((rows,), device=dev, dtype=torch.int32)
            if self.decode:
                device["row_seg"].copy_(torch.arange(rows, dtype=torch.int32))
                device["cu_rows"].copy_(torch.arange(rows + 1, dtype=torch.int32))
            else:
                device["row_seg"].fill_(-1)
            self.rows = H.Rows(positions=self.positions, row_seg=device["row_seg"], cu_rows=device["cu_rows"], page_table=self.page_table,
                               slots=device["slots"], decode=self.decode)
            self.synced_owner_state = None
            self.repeat_key: tuple | None = None
            self.repeat_tokens: list[int] = []
            self.repeat_left = 0
            self.repeat_version = -1
            self.program: list[Callable[[], None]] = []
            self.launches_per_step = 0
            self.cuda_graph = None
            self.feedback_graph = None
            self.h2d_done = torch.cuda.Event()
            self.steps_run = 0
            self.logits: torch.Tensor | None = None
            self._lower()

        # -- metadata ----------------------------------------------------------------------
        def sync_sessions(self, sessions: list[Any]) -> None:
            before = self.synced_owner_state
            super().sync_sessions(sessions)
            if before is None or [(s[0], s[3]) for s in before] != [(s[0], s[3]) for s in self.synced_owner_state]:
                slots = self._host["slots"]
                slots.numpy()[:] = [s.kv_cache.state_slot or 0 for s in sessions]
                self._device_slots.copy_(slots, non_blocking=True)

        def sync_portions(self, portions: list[tuple[Any, int, list[int]]], wanted_rows: list[int]) -> None:
            """Rows of this step: `portions` = (cache, first position, tokens) per sequence, pages reserved; `wanted_rows`
            are the rows whose logits the head computes. What is beyond them is padding."""
            self.h2d_done.synchronize()          # the pinned staging buffers must not change under a pending copy
            host = {k: v.numpy() for k, v in self._host.items()}
            ids, table = self.host_ids.numpy(), self.host_table.numpy()
            host["lens"][:] = 0
            host["row_seg"][:] = -1
            ids[:] = 0
            row = 0
            for seg, (cache, start, tokens) in enumerate(portions):
                n = len(tokens)
                ids[row:row + n] = tokens
                host["lens"][row:row + n] = np.arange(start, start + n)
                host["row_seg"][row:row + n] = seg
                host["cu_rows"][seg] = row
                host["slots"][seg] = cache.state_slot or 0
                table[seg] = cache.page_table_row(self.width)
                row += n
            host["cu_rows"][len(portions):] = row
            host["logit_index"][:] = 0
            host["logit_index"][:len(wanted_rows)] = wanted_rows
            self.ids.copy_(self.host_ids, non_blocking=True)
            self._meta.copy_(self._host_meta, non_blocking=True)
            self.h2d_done.record()

        # -- lowering ----------------------------------------------------------------------
        def _scratch(self, role: str, cols: int, dtype: torch.dtype | None = None, rows: int | None = None) -> torch.Tensor:
            """A [rows, cols] buffer from the engine's storage for `role`: plans run one after the other on one stream, and
            within a step a role is rewritten layer by layer."""
            dtype = self.engine.dtype if dtype is None else dtype
            rows = self.batch if rows is None else rows
            flat = self.engine.scratch(role, rows * cols * torch.empty((), dtype=dtype).element_size())
            return flat.view(dtype)[:rows * cols].view(rows, cols)

        def _dyt(self, names: list[str]) -> H.DynamicTanh:
            w = self.engine.weights
            return H.DynamicTanh(w.get_f32(names[0]), w.get_f32(names[1]), float(w.get_f32(names[2]).item()))

        def _next_after(self, idx: int) -> tuple[H.Next | None, str | None]:
            """What the kernel finishing the residual at node `idx` can leave for the node behind it."""
            nxt = self._nodes[idx + 1]
            width = int(self.engine.config.hidden_size)
            if nxt.op == "dynamic_tanh" and nxt.attrs.get("rows") != "logits" and nxt.inputs[0] == self._nodes[idx].outputs[0]:
                out = self._scratch("normed", width)
                return H.Next(out, self._dyt(nxt.inputs[1:4])), nxt.outputs[0]
            if nxt.op == "rms_norm" and nxt.attrs.get("rows") != "logits" and nxt.inputs[0] == self._nodes[idx].outputs[0]:
                norm = H.RmsNorm(self.engine.weights.get_f32(nxt.inputs[1]), float(nxt.attrs["eps"]))
                return H.Next(self._scratch("normed", width), norm), nxt.outputs[0]
            if nxt.op == "layer_norm" and nxt.attrs.get("rows") != "logits" and nxt.inputs[0] == self._nodes[idx].outputs[0]:
                norm = H.LayerNorm(self.engine.weights.get_f32(nxt.inputs[1]), float(nxt.attrs["eps"]))
                return H.Next(self._scratch("normed", width), norm), nxt.outputs[0]
            if nxt.op in READS_RESIDUAL and nxt.inputs[0] == self._nodes[idx].outputs[0]:
                return H.Next(self._scratch("copied", width)), None
            return None, None

        def _finish_residual(self, idx: int, emit: Callable[[H.Next | None], None]) -> None:
            """Emit the kernel that updates the residual at node `idx` and record its outputs."""
            nx, normed = self._next_after(idx)
            emit(nx)
            node = self._nodes[idx]
            self._env[node.outputs[0]] = self._residual
            if normed is not None:
                self._env[normed] = nx.out
                self._skip.add(idx + 1)
            elif nx is not None:
                self._env["copy:" + node.outputs[0]] = nx.out

        def _lower(self) -> None:
            eng = self.engine
            self._nodes = list(eng.graph.nodes)
            self._env: dict[str, Any] = {}
            self._skip: set[int] = set()
            self._count_keys: list[tuple[str, int]] = []
            self._count_totals = None
            self._residual = self._scratch("residual", int(eng.config.hidden_size), torch.float32)
            self._emit(lambda: ops.advance_positions(self.positions, self.seq_lens), "b200.advance_positions")
            for idx, node in enumerate(self._nodes):
                if idx in self._skip:
                    continue
                lower = getattr(self, "_lower_" + node.op, None)
                if lower is None:
                    raise NotImplementedError(f"ragged plans do not implement op {node.op}")
                lower(idx, node)
            logits = self._env[eng.graph.outputs[0]]
            self.logits = logits
            self.feedback_tail = lambda: ops.argmax_rows(logits, self.ids)

        def _dense(self, x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bias: torch.Tensor | None = None, label: str = "",
                   relu2: bool = False) -> None:
            """Plain product into `out` (float32 for logits), or its squared ReLU: tensor cores where they take it, else CUDA cores."""
            if H.dense_supported(int(w.shape[1]), w.stride(0), x.stride(0), dtype=x.dtype):
                epilogue = H.DENSE_RELU2 if relu2 else H.DENSE_F32 if out.dtype == torch.float32 else H.DENSE_PLAIN
                self._emit(lambda: H.dense_gemm(x, w, out, epilogue=epilogue, bias=bias), "b200.dense_gemm" + label)
            else:
                self._emit(lambda: H.dense_simple(x, w, out, bias=bias), "b200.dense_simple")
                if relu2:
                    self._emit(lambda: H.relu2_cols(out, int(w.shape[0])), "b200.relu2_cols")

        def _input(self, name: str) -> torch.Tensor:
            """A product's input: an activation, or the residual's copy."""
            return self._env.get("copy:" + name, self._env[name])

        def _lower_scaled_token_embedding(self, idx: int, node: Any) -> None:
            table = self.engine.weights.get_checked(node.inputs[1])
            scale, x = float(node.attrs["scale"]), self._residual
            self._finish_residual(idx, lambda nx: self._emit(lambda: H.scaled_embedding(table, self.ids, x, scale, nx), "b200.scaled_embedding"))

        def _lower_add_token_embedding(self, idx: int, node: Any) -> None:
            """The embedding output once more, from the table."""
            table = self.engine.weights.get_checked(node.inputs[2])
            scale, x = float(node.attrs["scale"]), self._residual
            self._finish_residual(idx, lambda nx: self._emit(lambda: H.scaled_embedding(table, self.ids, x, scale, nx, accumulate=True),
                                                             "b200.add_embedding"))

        def _lower_join_embedding(self, idx: int, node: Any) -> None:
            """residual = product of (residual, embedding output) + one row of the last input."""
            eng, x = self.engine, self._residual
            table, w = eng.weights.get_checked(node.inputs[2]), eng.weights.get_checked(node.inputs[3])
            step = eng.weights.get_f32(node.inputs[4])[int(node.attrs["step"])]
            joined = self._scratch("joined", int(w.shape[1]))
            self._emit(lambda: H.join_embedding(x, table, self.ids, joined), "b200.join_embedding")
            self._dense(joined, w, x, step, ".join")
            self._env[node.outputs[0]] = x

        def _lower_dynamic_tanh(self, idx: int, node: Any) -> None:
            norm = self._dyt(node.inputs[1:4])
            width = int(self.engine.config.hidden_size)
            if node.attrs.get("rows") == "logits":
                out = self._scratch("final", width, rows=self.logit_rows)
                self._emit(lambda: H.dyt_rows(self._residual, norm, out, self.logit_index), "b200.dyt_rows")
            else:
                out = self._scratch("normed", width)
                self._emit(lambda: H.dyt_rows(self._residual, norm, out), "b200.dyt_rows")
            self._env[node.outputs[0]] = out

        def _lower_concat_matmul(self, idx: int, node: Any) -> None:
            eng, x = self.engine, self._input(node.inputs[0])
            names = tuple(node.inputs[1:])
            bias = eng.concat_bias(tuple(node.attrs["bias"]), names) if node.attrs.get("bias") else None
            sizes = list(node.attrs.get("sizes") or [int(eng.graph.weights[n].shape[0]) for n in names])      # outputs, by default one per weight
            w = eng.concat_weight(names)
            floats = sum(sizes[len(sizes) - int(node.attrs.get("float_tail", 0)):])     # the last columns: float32, one output
            total = int(w.shape[0]) - floats
            out = self._scratch("projected", (total + 7) // 8 * 8)
            tail = self._scratch("projected_float", floats, torch.float32) if floats else None
            act = sum(sizes[: int(node.attrs.get("activated", 0))])
            if H.dense_supported(int(w.shape[1]), w.stride(0), x.stride(0), dtype=x.dtype):
                epilogue = H.DENSE_SILU if act else H.DENSE_PLAIN
                self._emit(lambda: H.dense_gemm(x, w, out, epilogue=epilogue, act_cols=act, bias=bias, tail=tail),
                           "b200.dense_gemm" + (".silu" if act else ""))
            else:
                main, main_bias = w[:total], None if bias is None else bias[:total]
                self._emit(lambda: H.dense_simple(x, main, out, bias=main_bias), "b200.dense_simple")
                if tail is not None:
                    rest, rest_bias = w[total:], None if bias is None else bias[total:]
                    self._emit(lambda: H.dense_simple(x, rest, tail, bias=rest_bias), "b200.dense_simple")
                if act:
                    self._emit(lambda: H.silu_cols(out, act), "b200.silu_cols")
            col = 0
            if tail is not None:
                self._env[node.outputs[-1]] = tail
                sizes = sizes[:len(sizes) - int(node.attrs["float_tail"])]
            for name, n in zip(node.outputs, sizes):
                self._env[name] = out[:, col:col + n]
                col += n

        def _lower_latent_attention(self, idx: int, node: Any) -> None:
            eng, at = self.engine, node.attrs
            q, gate = self._env[node.inputs[0]], self._env[node.inputs[1]]
            uk, uv = eng.weights.get_checked(node.inputs[2]), eng.weights.get_checked(node.inputs[3])
            sink = eng.weights.get_f32(node.inputs[4])
            down = self._env[node.inputs[5]] if len(node.inputs) > 5 else None
            down_norm = eng.weights.get_f32(node.inputs[6]) if len(node.inputs) > 6 else None
            heads, dim, rot, vdim, rank = (int(at[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            pool = eng.allocator.pool_for_layer(int(at["cache_layer"]))["latent"]
            table = eng.rotate_half_table(int(at["rot_dims"]), float(at["rot_base"]))
            args = H.latent_args(self.rows, pool, heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, window=int(at["window"]),
                                 scale=float(at["scale"]))
            out = self._scratch("mixed", heads * vdim)
            fast = (H.latent_attention_supported(rank, rot, eng.page_size, eng.dtype) and dim % 8 == 0
                    and H.dense_supported(dim, dim, q.stride(0), dtype=q.dtype, batch=heads, x_batch_cols=dim + rot)
                    and H.dense_supported(rank, rank, heads * rank, dtype=q.dtype, batch=heads, x_batch_cols=rank))
            if fast:
                q_lat = self._scratch("latent_q", heads * (rank + rot))
                q_rot, head_stride = q_lat[:, rank:], rank + rot
            else:
                q_rot, head_stride = q[:, dim:], dim + rot           # turned in place
            self._emit(lambda: H.latent_prepare(args, q, q_rot, q_rot_head_stride=head_stride, table=table, rot_dims=int(at["rot_dims"]),
                                                down=down, norm_weight=down_norm, eps=float(at["eps"])), "b200.latent_prepare")
            if not fast:
                self._emit(lambda: H.latent_attention_simple(args, q, uk, uv, sink, gate, out), "b200.latent_attention_simple")
                self._env[node.outputs[0]] = out
                return
            # key up-projection absorbed into the queries, attention over latents, value up-projection with the output gate
            uk_t = eng.absorbed_weight(node.inputs[2], heads, dim, rank)
            o_lat = self._scratch("latent_o", heads * rank)
            splits = H.latent_attention_splits(self.batch, heads, int(at["window"]), self.width, eng.page_size) if self.decode else 1
            self._emit(lambda: H.dense_gemm(q, uk_t, q_lat, batch=heads, x_batch_cols=dim + rot, y_batch_cols=rank + rot), "b200.dense_gemm.heads")
            self._emit(lambda: H.latent_attention(args, q_lat, sink, o_lat, splits=splits), "b200.latent_attention")
            self._emit(lambda: H.dense_gemm(o_lat, uv, out, epilogue=H.DENSE_GATED, batch=heads, x_batch_cols=rank, gate=gate),
                       "b200.dense_gemm.heads_gated")
            self._env[node.outputs[0]] = out

        def _lower_linear_recurrence(self, idx: int, node: Any) -> None:
            eng, at = self.engine, node.attrs
            q, k, v = (self._env[n] for n in node.inputs)
            heads, dim, vdim = int(at["heads"]), int(at["dim"]), int(at["vdim"])
            state = eng.allocator.state_for_layer(int(at["layer"]))
            out = self._scratch("recurrence", heads * vdim)
            args = H.recurrence_args(self.rows, q, k, v, eng.decay_powers(tuple(at["decay"])), state, out, heads=heads, dim=dim, vdim=vdim)
            if self.decode and vdim % 4 == 0 and vdim <= 1024:
                self._emit(lambda: H.recurrence_step(args), "b200.recurrence_step")
            elif H.recurrence_chunked_supported(dim, vdim, eng.dtype) and q.stride(0) % 8 == 0:
                need = H.recurrence_workspace_bytes(self.batch, self.segments, heads, dim, vdim)
                ws = eng.scratch("recurrence_ws", need) if need else None
                self._emit(lambda: H.recurrence_chunked(args, ws), "b200.recurrence_chunked", launches=3 if need else 1)
            else:
                self._emit(lambda: H.recurrence_simple(args), "b200.recurrence_simple")
            self._env[node.outputs[0]] = out

        def _lower_matrix_memory(self, idx: int, node: Any) -> None:
            eng, at = self.engine, node.attrs
            q, k, v, logits, gate = (self._env[n] for n in node.inputs[:5])
            in_bias, forget_bias, norm = (eng.weights.get_f32(n) for n in node.inputs[5:8])
            heads, dim, vdim, eps = int(at["heads"]), int(at["dim"]), int(at["vdim"]), float(at["eps"])
            state = eng.allocator.state_for_layer(int(at["layer"]))
            gates = H.MemoryGates(logits, in_bias, forget_bias, float(at["gate_cap"]))
            mixed, scale = self._scratch("memory_mixed", heads * vdim), float(dim) ** -0.5
            self._env[node.outputs[0]] = mixed
            if self.decode and vdim % 4 == 0 and vdim <= 1024 and dim <= 4096:
                args = H.recurrence_args(self.rows, q, k, v, None, state, mixed, heads=heads, dim=dim, vdim=vdim, q_scale=scale)
                self._emit(lambda: H.memory_step(args, gates, gate, norm, eps), "b200.memory_step")
                return
            log_decay, log_take, maximum, normaliser = (self._scratch("memory_" + role, heads, torch.float32)
                                                        for role in ("decay", "take", "maximum", "normaliser"))
            out = self._scratch("recurrence", heads * vdim)
            args = H.recurrence_args(self.rows, q, k, v, None, state, out, heads=heads, dim=dim, vdim=vdim, gated=(log_decay, log_take, normaliser),
                                     q_scale=scale)
            self._emit(lambda: H.memory_gates(args, gates, log_decay, log_take, maximum), "b200.memory_gates")
            aligned = q.stride(0) % 8 == 0 and not any(t.data_ptr() % 16 for t in (q, k, v))
            if H.recurrence_chunked_supported(dim, vdim, eng.dtype) and aligned:
                need = H.recurrence_workspace_bytes(self.batch, self.segments, heads, dim, vdim)
                ws = eng.scratch("recurrence_ws", need) if need else None
                self._emit(lambda: H.recurrence_chunked(args, ws), "b200.recurrence_chunked", launches=3 if need else 1)
            else:
                self._emit(lambda: H.recurrence_simple(args), "b200.recurrence_simple")
            self._emit(lambda: H.memory_norm(out, normaliser, maximum, gate, norm, eps, mixed, heads=heads, vdim=vdim), "b200.memory_norm")

        def _lower_short_conv(self, idx: int, node: Any) -> None:
            """Inputs: x, bias by name or "", convolution weights of neighbouring channels. One output per attrs["sizes"]."""
            eng, x = self.engine, self._env[node.inputs[0]]
            w = eng.concat_f32(tuple(node.inputs[2:]))
            bias = eng.weights.get_f32(node.inputs[1]) if node.inputs[1] else None
            state, offset = eng.allocator.state_for_layer(int(node.attrs["layer"])), int(node.attrs["offset"])
            channels = int(w.shape[0])
            out = self._scratch("convolved", (channels + 7) // 8 * 8)[:, :channels]
            self._emit(lambda: M.short_conv(self.rows, x, w, bias, state, offset, out), "b200.short_conv")
            col = 0
            for name, n in zip(node.outputs, node.attrs["sizes"]):
                self._env[name] = out[:, col:col + n]
                col += n

        def _lower_state_space(self, idx: int, node: Any) -> None:
            eng, at = self.engine, node.attrs
            q, k, v, logits = (self._env[n] for n in node.inputs[:4])
            bias, log_rate, skip = (eng.weights.get_f32(n) for n in node.inputs[4:7])
            heads, key_heads, dim, vdim = (int(at[n]) for n in ("heads", "key_heads", "dim", "vdim"))
            state = eng.allocator.state_for_layer(int(at["layer"]))
            steps = H.StepSizes(logits, bias, log_rate)
            out = self._scratch("recurrence", heads * vdim)
            self._env[node.outputs[0]] = out

            def args(gated: tuple | None) -> Any:
                return H.recurrence_args(self.rows, q, k, v, None, state, out, heads=heads, dim=dim, vdim=vdim, gated=gated, key_heads=key_heads,
                                         skip=skip, memory=False)
            if self.decode and vdim % 4 == 0 and vdim <= 1024 and dim <= 4096:
                a = args(None)
                self._emit(lambda: H.state_space_step(a, steps), "b200.state_space_step")
                return
            log_decay, log_take = (self._scratch("space_" + role, heads, torch.float32) for role in ("decay", "take"))
            a = args((log_decay, log_take, None))
            self._emit(lambda: H.state_space_gates(a, steps, log_decay, log_take), "b200.state_space_gates")
            aligned = q.stride(0) % 8 == 0 and not any(t.data_ptr() % 16 for t in (q, k, v))
            if H.recurrence_chunked_supported(dim, vdim, eng.dtype) and aligned:
                need = H.recurrence_workspace_bytes(self.batch, self.segments, heads, dim, vdim)
                ws = eng.scratch("recurrence_ws", need) if need else None
                self._emit(lambda: H.recurrence_chunked(a, ws), "b200.recurrence_chunked", launches=3 if need else 1)
            else:
                self._emit(lambda: H.recurrence_simple(a), "b200.recurrence_simple")

        def _lower_delta_rule(self, idx: int, node: Any) -> None:
            """Inputs: q, k, v, gate logits, output gate, then bias and log rate of the decay and the head's norm weight."""
            eng, at = self.engine, node.attrs
            q, k, v, logits, gate = (self._env[n] for n in node.inputs[:5])
            bias, log_rate, norm = (eng.weights.get_f32(n) for n in node.inputs[5:8])
            heads, key_heads, dim, vdim, eps = int(at["heads"]), int(at["key_heads"]), int(at["dim"]), int(at["vdim"]), float(at["eps"])
            state = eng.allocator.state_for_layer(int(at["layer"]))
            mixed = self._scratch("mixed", heads * vdim)
            self._env[node.outputs[0]] = mixed

            def args(out: torch.Tensor) -> Any:
                return M.delta_args(self.rows, q, k, v, logits, bias, log_rate, state, out, heads=heads, key_heads=key_heads, dim=dim, vdim=vdim)
            if self.decode and vdim % 4 == 0 and vdim <= 1024 and dim <= 4096:
                a = args(mixed)
                self._emit(lambda: M.delta_step(a, gate, norm, eps), "b200.delta_step")
                return
            out = self._scratch("recurrence", heads * vdim)
            a = args(out)
            aligned = q.stride(0) % 8 == 0 and not any(t.data_ptr() % 16 for t in (q, k, v))
            if M.delta_chunked_supported(dim, vdim, eng.dtype) and aligned:
                ws = eng.scratch("delta_ws", M.delta_workspace_bytes(self.batch, self.segments, heads))
                self._emit(lambda: M.delta_chunked(a, ws), "b200.delta_chunked", launches=2)
            else:
                self._emit(lambda: M.delta_simple(a), "b200.delta_simple")
            self._emit(lambda: H.gated_parts_rms(out, gate, norm, eps, mixed, parts=heads, gate_first=False), "b200.gated_parts_rms")

        def _lower_gated_parts_rms(self, idx: int, node: Any) -> None:
            o, gate = self._env[node.inputs[0]], self._env[node.inputs[1]]
            w, eps = self.engine.weights.get_f32(node.inputs[2]), float(node.attrs["eps"])
            parts, first = int(node.attrs["parts"]), bool(node.attrs["gate_first"])
            out = self._scratch("mixed", int(o.shape[1]))
            self._emit(lambda: H.gated_parts_rms(o, gate, w, eps, out, parts=parts, gate_first=first), "b200.gated_parts_rms")
            self._env[node.outputs[0]] = out

        def _lower_gated_rms_norm(self, idx: int, node: Any) -> None:
            o, gate = self._env[node.inputs[0]], self._env[node.inputs[1]]
            w, eps = self.engine.weights.get_f32(node.inputs[2]), float(node.attrs["eps"])
            out = self._scratch("mixed", int(o.shape[1]))
            self._emit(lambda: H.gated_rms(o, gate, w, eps, out), "b200.gated_rms")
            self._env[node.outputs[0]] = out

        def _lower_matmul(self, idx: int, node: Any) -> None:
            eng, x = self.engine, self._env[node.inputs[0]]
            w = eng.weights.get_checked(node.inputs[1])
            nxt = self._nodes[idx + 1] if idx + 1 < len(self._nodes) else None
            if (nxt is not None and nxt.op == "residual_dynamic_tanh" and nxt.inputs[1] == node.outputs[0]
                    and H.dense_supported(int(w.shape[1]), w.stride(0), x.stride(0), dtype=x.dtype)):
                norm, res = self._dyt(nxt.inputs[2:5]), self._residual
                self._finish_residual(idx + 1, lambda nx: self._emit(
                    lambda: H.dense_gemm(x, w, epilogue=H.DENSE_RESIDUAL, residual=res, norm=norm, nx=nx), "b200.dense_gemm.residual_dyt"))
                self._skip.add(idx + 1)
                return
            if nxt is None:
                out = self._scratch("logits", int(w.shape[0]), torch.float32, rows=self.logit_rows)
            else:
                out = self._scratch(str(node.attrs.get("role", "sublayer")), int(w.shape[0]))      # (a shared expert's lives until the combine)
            bias = node.attrs.get("bias")
            self._dense(x, w, out, None if bias is None else eng.weights.get_f32(bias), "." + str(node.attrs["projection"]),
                        relu2=node.attrs.get("activation") == "relu2")
            self._env[node.outputs[0]] = out

        def _lower_residual_dynamic_tanh(self, idx: int, node: Any) -> None:
            y, norm, res = self._env[node.inputs[1]], self._dyt(node.inputs[2:5]), self._residual
            self._finish_residual(idx, lambda nx: self._emit(lambda: H.residual_dyt(res, y, norm, nx), "b200.residual_dyt"))

        def _lower_fused_geglu(self, idx: int, node: Any) -> None:
            self._env[node.outputs[0]] = self._glu(self._env[node.inputs[0]], node, "gelu_tanh")

        def _lower_fused_glu(self, idx: int, node: Any) -> None:
            self._env[node.outputs[0]] = self._glu(self._input(node.inputs[0]), node, node.attrs["activation"])

        def _glu(self, x: torch.Tensor, node: Any, activation: str, tail_weights: tuple[str, ...] = (),
                 tail: torch.Tensor | None = None) -> torch.Tensor:
            """activation(gate, up) of one product; rows of `tail_weights` behind the pairs leave plain float32 columns."""
            eng = self.engine
            names = tuple(node.inputs[1:3])
            w = eng.paired_weight(names, tail_weights)
            ff = int(eng.graph.weights[names[0]].shape[0])
            bias = eng.paired_bias(tuple(node.attrs["bias"])) if node.attrs.get("bias") else None
            kind, limit = H.GLU_EPILOGUES[activation], float(node.attrs.get("limit", 0.0))
            out = self._scratch("gated", (ff + 7) // 8 * 8)[:, :ff]
            if H.dense_supported(int(w.shape[1]), w.stride(0), x.stride(0), dtype=x.dtype):
                label = GLU_LABELS[activation]
                self._emit(lambda: H.dense_gemm(x, w, out, epilogue=kind, bias=bias, limit=limit, tail=tail), "b200.dense_gemm" + label)
            else:
                both, out = self._scratch("gate_up", 2 * ff), self._scratch("gated", ff)
                self._emit(lambda: H.dense_simple(x, w, both, bias=bias), "b200.dense_simple")
                self._emit(lambda: H.glu_pairs(both, out, kind, limit), "b200.glu_pairs")
            return out

        def _lower_token_side_gate(self, idx: int, node: Any) -> None:
            eng = self.engine
            x = self._env["copy:" + node.inputs[0]]
            w, table = eng.weights.get_checked(node.inputs[1]), eng.weights.get_checked(node.inputs[2])
            dim, col = int(w.shape[0]), int(node.attrs["column"])
            out = self._scratch("side", dim)
            if H.dense_supported(int(w.shape[1]), w.stride(0), x.stride(0), dtype=x.dtype):
                self._emit(lambda: H.dense_gemm(x, w, out, epilogue=H.DENSE_GELU_EMBED, ids=self.ids, table=table, table_col=col),
                           "b200.dense_gemm.gelu_embed")
            else:
                g = self._scratch("side_gate", dim)
                self._emit(lambda: H.dense_simple(x, w, g), "b200.dense_simple")
                self._emit(lambda: H.gelu_embed(g, self.ids, table, col, out), "b200.gelu_embed")
            self._env[node.outputs[0]] = out

        def _lower_residual_rms_norm(self, idx: int, node: Any) -> None:
            y, res = self._env[node.inputs[1]], self._residual
            w, eps = self.engine.weights.get_f32(node.inputs[2]), float(node.attrs["eps"])
            self._finish_residual(idx, lambda nx: self._emit(lambda: H.residual_rms(res, y, w, eps, nx), "b200.residual_rms"))

        def _lower_residual_add(self, idx: int, node: Any) -> None:
            y, res = self._env[node.inputs[1]], self._residual
            scale = self.engine.weights.get_f32(node.inputs[2]) if len(node.inputs) > 2 else None
            self._finish_residual(idx, lambda nx: self._emit(lambda: H.residual_add(res, y, nx, scale), "b200.residual_add"))

        def _lower_residual_rms_pair(self, idx: int, node: Any) -> None:
            y1, y2, res = self._env[node.inputs[1]], self._env[node.inputs[3]], self._residual
            w1, w2 = (self.engine.weights.get_f32(node.inputs[i]) for i in (2, 4))
            factor, eps = float(node.attrs["factor"]), float(node.attrs["eps"])
            self._finish_residual(idx, lambda nx: self._emit(lambda: H.residual_rms_pair(res, y1, w1, y2, w2, factor, eps, nx),
                                                             "b200.residual_rms_pair"))

        def _lower_rms_norm(self, idx: int, node: Any) -> None:
            w, eps = self.engine.scaled_weight(node.inputs[1], float(node.attrs.get("scale", 1.0))), float(node.attrs["eps"])
            logits = node.attrs.get("rows") == "logits"
            out = self._scratch("final" if logits else "normed", int(w.numel()), rows=self.logit_rows if logits else None)
            index = self.logit_index if logits else None
            self._emit(lambda: H.rms_rows(self._residual, w, eps, out, index), "b200.rms_rows")
            self._env[node.outputs[0]] = out

        def _lower_layer_norm(self, idx: int, node: Any) -> None:
            w, eps = self.engine.weights.get_f32(node.inputs[1]), float(node.attrs["eps"])
            logits = node.attrs.get("rows") == "logits"
            out = self._scratch("final" if logits else "normed", int(w.numel()), rows=self.logit_rows if logits else None)
            index = self.logit_index if logits else None
            self._emit(lambda: H.layer_norm_rows(self._residual, w, eps, out, index), "b200.layer_norm_rows")
            self._env[node.outputs[0]] = out

        def _lower_talking_attention(self, idx: int, node: Any) -> None:
            eng, at = self.engine, node.attrs
            q, k, v = (self._env[n] for n in node.inputs[:3])
            heads, kv_heads, dim, vdim, rot = (int(at[n]) for n in ("heads", "kv_heads", "dim", "vdim", "rot_dims"))
            pool = eng.allocator.pool_for_layer(int(at["layer"]))
            yarn = at.get("yarn")
            table = None
            if rot:
                table = eng.rotate_half_table(rot, float(at["rot_base"])) if yarn is None else eng.yarn_table(rot, float(at["rot_base"]), tuple(map(float, yarn)))
            args = M.talking_args(self.rows, pool["key_rows"], pool["value_rows"], eng.weights.get_f32(node.inputs[3]), heads=heads, kv_heads=kv_heads, dim=dim,
                                  vdim=vdim, window=int(at["window"]), scale=float(at["scale"]))
            shape = (heads, kv_heads, dim, vdim, eng.page_size, eng.dtype)
            step = self.decode and M.talking_step_supported(*shape)
            mixed = not step and M.talking_prompt_supported(*shape)
            prepared = self._scratch("prepared_q", heads * dim * (kv_heads if mixed else 1))
            out = self._scratch("mixed", heads * vdim)
            self._emit(lambda: M.talking_prepare(args, q, k, v, prepared, eps=float(at["eps"]), table=table, mixed=mixed), "b200.talking_prepare")
            if step:
                splits = M.talking_step_splits(self.batch, heads, kv_heads, dim, vdim, int(at["window"]), self.width, eng.page_size)
                self._emit(lambda: M.talking_step(args, prepared, out, splits=splits), "b200.talking_step")
            elif mixed:
                self._emit(lambda: M.talking_prompt(args, prepared, out), "b200.talking_prompt")
            else:
                self._emit(lambda: M.talking_simple(args, prepared, out), "b200.talking_simple")
            self._env[node.outputs[0]] = out

        def _lower_tied_attention(self, idx: int, node: Any) -> None:
            """Inputs: q, k, then by name or "" output gate, sink, values of their own, weights of the query and key norm."""
            eng, at = self.engine, node.attrs
            names = list(node.inputs) + [""] * (7 - len(node.inputs))
            q, k, gate, v = (self._env[n] if n else None for n in (names[0], names[1], names[2], names[4]))
            sink, q_weight, k_weight = (eng.weights.get_f32(n) if n else None for n in (names[3], names[5], names[6]))
            heads, kv_heads, dim, rot = (int(at[n]) for n in ("heads", "kv_heads", "dim", "rot_dims"))
            key_dim = None if v is None else int(at["key_dim"])
            whole = bool(at.get("whole_norm", False))
            pool = eng.allocator.pool_for_layer(int(at["layer"]))
            scaling = at.get("rot_scaling")
            table = eng.rotate_half_table(rot, float(at["rot_base"]), None if scaling is None else tuple(map(float, scaling))) if rot else None
            reach = float(dim if key_dim is None else key_dim)              # of unit root mean squares
            reach *= ((heads * kv_heads) ** 0.5 if whole else 1.0) * eng.largest_weight(names[5]) * eng.largest_weight(names[6])
            args = X.tied_args(self.rows, pool["rows"], pool["inv_rms"], heads=heads, kv_heads=kv_heads, dim=dim, rot_dims=rot,
                               window=int(at["window"]), keep_first=int(at["keep_first"]), scale=float(at["scale"]), softcap=at.get("softcap"),
                               sink=sink, key_dim=key_dim, reach=reach)
            prepared = self._scratch("prepared_q", heads * X.query_width(dim, rot, key_dim))
            out = self._scratch("mixed", heads * dim)
            self._emit(lambda: X.tied_prepare(args, q, k, prepared, eps=float(at["eps"]), table=table, v=v, q_weight=q_weight, k_weight=k_weight,
                                              whole=whole), "b200.tied_prepare")
            if self.decode and X.tied_step_supported(heads, kv_heads, dim, rot, eng.page_size, eng.dtype, key_dim):
                splits = X.tied_step_splits(self.batch, heads, kv_heads, int(at["window"]), int(at["keep_first"]), self.width, eng.page_size)
                self._emit(lambda: X.tied_attention_step(args, prepared, gate, out, splits=splits), "b200.tied_attention_step")
            elif (X.tied_prompt_supported(heads, kv_heads, dim, rot, eng.page_size, eng.dtype, key_dim)
                  and (gate is None or gate.stride(0) % 8 == 0)):
                self._emit(lambda: X.tied_attention_prompt(args, prepared, gate, out), "b200.tied_attention_prompt")
            else:
                self._emit(lambda: X.tied_attention_simple(args, prepared, gate, out), "b200.tied_attention_simple")
            self._env[node.outputs[0]] = out

        def _lower_expert_router(self, idx: int, node: Any) -> None:
            """Inputs: x, router, then by name or "" correction and the shared expert's gate (one row)."""
            eng, x, at = self.engine, self._input(node.inputs[0]), node.attrs
            names = list(node.inputs) + [""] * (4 - len(node.inputs))
            spec = eng.graph.weights[names[1]]
            scored, width, top, scale = int(spec.shape[0]), int(spec.shape[1]), int(at["top"]), float(at["scale"])
            identity = int(at.get("identity", 0))
            experts = scored - identity
            rule = None
            if at.get("scores") == "softmax":
                rule = X.SoftmaxRule(eng.weights.get_f32(names[2]) if names[2] else None, int(at["groups"]), int(at["keep"]), identity)
            rows_of = (names[1],) + ((names[3],) if names[3] else ())
            logits = self._scratch("router_logits", scored + len(rows_of) - 1, torch.float32)
            nxt = self._nodes[idx + 1]
            if (nxt.op == "fused_glu" and nxt.inputs[0] == node.inputs[0] and not nxt.attrs.get("bias")
                    and H.dense_supported(width, width, x.stride(0), dtype=x.dtype)):
                # a shared expert reads the same rows: the router's columns ride behind its gate and up
                self._env[nxt.outputs[0]] = self._glu(x, nxt, nxt.attrs["activation"], rows_of, logits)
                self._skip.add(idx + 1)
            else:
                self._dense(x, eng.concat_weight(rows_of), logits)
            i32 = torch.int32
            routing = X.Routing(experts, top, counters=self._scratch("route_counters", experts + 1, i32, rows=1).view(-1),
                                cu=self._scratch("route_cu", experts + 1, i32, rows=1).view(-1), token_of=self._scratch("route_token", top, i32).view(-1),
                                place_of=self._scratch("route_place", top, i32), chosen=self._scratch("route_chosen", top, i32),
                                weight=self._scratch("route_weight", top, torch.float32))
            placed = None
            if self.batch > X.grouped_all_rows() and X.grouped_supported(width, x.stride(0), eng.dtype):
                placed = self._scratch("placed", width, rows=routing.places)       # the experts' products read rows in expert order
            self._emit(lambda: X.route(logits, self.rows.row_seg, routing, scale, x, placed, rule), "b200.route", launches=1 if placed is None else 2)
            self._env[node.outputs[0]] = (routing, placed)
            if names[3]:
                self._env[node.outputs[1]] = logits[:, scored]

        def _lower_expert_mixture(self, idx: int, node: Any) -> None:
            eng, x = self.engine, self._input(node.inputs[0])
            routing, placed = self._env[node.inputs[1]]
            n = int(node.attrs["experts"])
            gates, ups, downs = (tuple(node.inputs[2 + i * n:2 + (i + 1) * n]) for i in range(3))
            w_in, w_out = eng.expert_pairs(gates, ups), eng.concat_weight(downs)
            ff, width = int(w_in.shape[0]) // (2 * n), int(w_out.shape[0]) // n
            activation = node.attrs["activation"]
            kind, limit = H.GLU_EPILOGUES[activation], float(node.attrs.get("limit", 0.0))
            places = routing.places
            out = self._scratch("expert_out", width, rows=places)
            if X.grouped_supported(int(w_in.shape[1]), x.stride(0), eng.dtype) and X.grouped_supported(ff, ff, eng.dtype):
                hidden = self._scratch("expert_hidden", ff, rows=places)
                source = x if placed is None else placed
                self._emit(lambda: X.grouped_gemm(source, w_in, hidden, routing, by_row=placed is None, epilogue=kind, limit=limit),
                           "b200.grouped_gemm" + GLU_LABELS[activation])
                self._emit(lambda: X.grouped_gemm(hidden, w_out, out, routing, by_row=False), "b200.grouped_gemm")
            else:
                both, hidden = self._scratch("expert_gate_up", 2 * ff, rows=places), self._scratch("expert_hidden", ff, rows=places)
                self._emit(lambda: X.grouped_simple(x, w_in, both, routing, gather=True), "b200.grouped_simple")
                self._emit(lambda: H.glu_pairs(both, hidden, kind, limit), "b200.glu_pairs")
                self._emit(lambda: X.grouped_simple(hidden, w_out, out, routing, gather=False), "b200.grouped_simple")
            self._env[node.outputs[0]] = out

        def _lower_combine_residual_rms_norm(self, idx: int, node: Any) -> None:
            y, (routing, _), res = self._env[node.inputs[1]], self._env[node.inputs[2]], self._residual
            w, eps = self.engine.weights.get_f32(node.inputs[3]), float(node.attrs["eps"])
            shared = self._env[node.inputs[4]] if len(node.inputs) > 4 else None
            self._finish_residual(idx, lambda nx: self._emit(lambda: X.combine_residual_rms(res, y, routing, shared, w, eps, nx),
                                                             "b200.combine_residual_rms"))

        def _lower_combine_residual(self, idx: int, node: Any) -> None:
            """Inputs: residual, experts' rows, routing, the experts' input, then the shared expert's output and its gate."""
            y, (routing, _), x, res = self._env[node.inputs[1]], self._env[node.inputs[2]], self._input(node.inputs[3]), self._residual
            shared, gate = (self._env[node.inputs[i]] if len(node.inputs) > i else None for i in (4, 5))
            self._finish_residual(idx, lambda nx: self._emit(lambda: X.combine_residual(res, y, routing, x, shared, gate, nx),
                                                             "b200.combine_residual"))

    return RaggedPlan
