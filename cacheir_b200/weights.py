"""Weight stores: load tensors by key, pack them on the GPU, cache by value name.

Mirrors `WeightStore` (cacheir/runtime/cpu.py:18-79) and `CudaWeightStore`
(cacheir/runtime/cuda.py:49-94): `get(name)` returns a dense tensor in the
runtime dtype (2-D weights are quantize->dequantize simulated when the
artifact is quantized, cpu.py:34-35); `get_quantized(name)` returns the packed
form. The pack itself runs on the device (`quantization.pack_weight_device`).
"""
from __future__ import annotations

import json
import struct
from pathlib import Path
from typing import Any, Callable, Mapping

import numpy as np
import torch

from .quantization import B200PackedWeight, dequantize_device, pack_weight_device


_SAFETENSORS_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16,
                       "I64": torch.int64, "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8,
                       "BOOL": torch.bool}


class SafetensorsFile:
    """A .safetensors file: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
    data_offsets), then the data. Tensors are CPU views of a private memory map."""

    def __init__(self, path: str | Path):
        self.path = Path(path)
        with open(self.path, "rb") as f:
            head = f.read(8)
            if len(head) != 8:
                raise ValueError(f"{self.path}: not a safetensors file")
            size = struct.unpack("<Q", head)[0]
            if size > self.path.stat().st_size - 8:
                raise ValueError(f"{self.path}: the header is longer than the file")
            self.entries: dict[str, dict] = json.loads(f.read(size))
        self.entries.pop("__metadata__", None)
        self._data = np.memmap(self.path, dtype=np.uint8, mode="c", offset=8 + size) if self.entries else np.empty(0, np.uint8)

    def __contains__(self, key: str) -> bool:
        return key in self.entries

    def tensor(self, key: str) -> torch.Tensor:
        entry = self.entries[key]
        begin, end = entry["data_offsets"]
        dtype = _SAFETENSORS_DTYPES[entry["dtype"]]
        shape = tuple(int(n) for n in entry["shape"])
        count = int(np.prod(shape, dtype=np.int64))
        if end - begin != count * torch.empty((), dtype=dtype).element_size() or end > self._data.size:
            raise ValueError(f"{self.path}: tensor {key!r} does not fit its data")
        raw = torch.from_numpy(np.array(self._data[begin:end]))     # (a copy: views of the map need not be aligned)
        return raw.view(dtype).reshape(shape) if count else torch.empty(shape, dtype=dtype)


class TensorSource:
    """Where raw tensors come from: an .npz or .safetensors file, a directory with one, a mapping key -> array,
    or a callable key -> tensor (synthetic weights generated on the device)."""

    def __init__(self, source: str | Path | Mapping[str, Any] | Callable[[str, tuple[int, ...]], torch.Tensor]):
        self._npz: dict[str, np.ndarray] | None = None
        self._mapping: Mapping[str, Any] | None = None
        self._callable = None
        self._path: Path | None = None
        self._safetensors: SafetensorsFile | None = None
        if callable(source):
            self._callable = source
        elif isinstance(source, Mapping):
            self._mapping = source
        else:
            self._path = Path(source)

    def load(self, key: str, shape: tuple[int, ...], file: str | None) -> Any:
        if self._callable is not None:
            return self._callable(key, shape)
        if self._mapping is not None:
            return self._mapping[key]
        path = self._path
        assert path is not None
        archive = path if path.suffix == ".safetensors" else path / "model.safetensors"
        if self._safetensors is None and archive.is_file() and not ((file or "").endswith(".npz") and (path / file).exists()):
            self._safetensors = SafetensorsFile(archive)
        if self._safetensors is not None:
            return self._safetensors.tensor(key)
        if path.is_file() and path.suffix == ".npz":
            npz_path = path
        elif path.is_dir():
            npz_path = path / (file or "weights.npz")
        else:
            raise FileNotFoundError(f"could not load weight {key!r} from {path}")
        if npz_path.suffix != ".npz" or not npz_path.exists():
            raise FileNotFoundError(f"cacheir_b200 loads .npz or .safetensors weights; {npz_path} not found")
        if self._npz is None:
            with np.load(npz_path) as data:
                self._npz = {k: data[k] for k in data.files}
        return self._npz[key]


class B200WeightStore:
    def __init__(self, source: TensorSource, specs: Mapping[str, Any], quant: str | None, *, device: torch.device,
                 dtype: torch.dtype):
        self.source = source
        self.specs = specs
        self.quant = quant
        self.device = device
        self.dtype = dtype
        self._cache: dict[str, torch.Tensor] = {}
        self._f32: dict[str, torch.Tensor] = {}
        self._qcache: dict[str, B200PackedWeight] = {}

    def _raw_fp32(self, value_name: str) -> torch.Tensor:
        spec = self.specs[value_name]
        shape = tuple(getattr(spec, "shape", None) or getattr(getattr(spec, "tensor_type", None), "shape", ()) or ())
        raw = self.source.load(spec.key, shape, getattr(spec, "file", None))
        if isinstance(raw, torch.Tensor):
            return raw.to(device=self.device, dtype=torch.float32)
        raw = np.array(raw, dtype=np.float32, order="C")        # (a scalar stays 0-dimensional)
        return torch.from_numpy(raw).to(self.device)

    def get(self, value_name: str) -> torch.Tensor:
        if value_name not in self._cache:
            tensor = self._raw_fp32(value_name)
            if self.quant and tensor.dim() == 2:
                # quantize -> dequantize simulation of a non-matmul 2-D weight; the pack is not kept
                packed = pack_weight_device(tensor.contiguous(), self.quant)
                if packed is None:
                    raise ValueError(f"Unsupported quantization mode {self.quant!r}")
                tensor = dequantize_device(packed, self.dtype)
            self._cache[value_name] = tensor.to(self.dtype).contiguous()
        return self._cache[value_name]

    def get_f32(self, value_name: str) -> torch.Tensor:
        """A parameter that stays in float32 whatever the runtime dtype is (norm weights, sinks, scalars)."""
        if value_name not in self._f32:
            self._f32[value_name] = self._checked(value_name).contiguous()
        return self._f32[value_name]

    def _checked(self, value_name: str) -> torch.Tensor:
        tensor = self._raw_fp32(value_name)
        want = tuple(self.specs[value_name].shape)
        if tuple(tensor.shape) != want:
            raise ValueError(f"weight {value_name!r} has shape {tuple(tensor.shape)}, the configuration needs {want}")
        return tensor

    def get_checked(self, value_name: str) -> torch.Tensor:
        """`get` of a weight whose shape the model's configuration fixes."""
        if value_name not in self._cache:
            self._cache[value_name] = self._checked(value_name).to(self.dtype).contiguous()
        return self._cache[value_name]

    def get_quantized(self, value_name: str) -> B200PackedWeight:
        if value_name not in self._qcache:
            tensor = self._raw_fp32(value_name)
            if tensor.dim() != 2:
                raise ValueError(f"Weight {value_name!r} is not a 2D matrix and cannot be packed")
            self._pack(value_name, tensor)
        return self._qcache[value_name]

    def _pack(self, value_name: str, tensor: torch.Tensor) -> B200PackedWeight:
        if value_name not in self._qcache:
            packed = pack_weight_device(tensor.contiguous(), self.quant)
            if packed is None:
                raise ValueError(f"Unsupported quantization mode {self.quant!r}")
            self._qcache[value_name] = packed
        return self._qcache[value_name]

    def put_quantized(self, value_name: str, packed: B200PackedWeight) -> None:
        """Install an already packed weight (e.g. group-wise int4 codes made elsewhere)."""
        self._qcache[value_name] = packed

    def release(self, value_name: str) -> None:
        """Forget the cached copies of a weight (its owner keeps a fused form)."""
        self._cache.pop(value_name, None)
        self._f32.pop(value_name, None)
        self._qcache.pop(value_name, None)
