"""A model directory (``config.json`` + ``*.safetensors`` [+ ``tokenizer.json``]) behind the interface of ``ZSELoader``.

The engine, the CLI and the server take a ``.zse`` file or such a directory; the runtime sees the same configuration,
weight index and tensor views either way.  Unquantised tensors are presented at the width their architecture is served
in: architectures that keep their checkpoints' bfloat16 (``ArchAdapter.STORED_DTYPE``) are views of the mapped file, the
others are rounded to fp16 as the converter would.  Tensors are copied to the device one by one; the streamed load needs
the contiguous weight section of a ``.zse`` file.
"""
from __future__ import annotations

import json
import os
from typing import Dict, Optional, Tuple

import numpy as np

from .arch import detect_architecture, get_adapter
from .config import ModelConfig
from .convert import _Shards, _to_f32, build_tensor_map, find_safetensor_files, round_bf16
from .loader import ZSELoader
from .spec import QuantMethod
from .weight_index import WeightEntry, WeightIndex

_INTEGER = {"I32": ("int32", 4), "I64": ("int32", 4)}
_WIDTH = {"float16": 2, "bfloat16": 2, "int32": 4}


class DirectoryLoader(ZSELoader):
    streamable = False

    def __init__(self, path: str):
        self._path = path
        self._fd, self._mm = None, None
        with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as f:
            raw = json.load(f)
        adapter = get_adapter(detect_architecture(raw))
        self._config: ModelConfig = adapter.config_from_hf(raw)
        self._config.quant.method, self._config.quant.bits = int(QuantMethod.NONE), 16
        self._source: Dict[str, Tuple[str, dict, int]] = {}
        self._weight_index = WeightIndex()
        self._shards = _Shards()
        tensors = build_tensor_map(find_safetensor_files(path))
        for name in adapter.tensor_load_order(list(tensors)):
            src = tensors[name]
            info = src[1]
            dtype = _INTEGER[info["dtype"]][0] if info["dtype"] in _INTEGER else adapter.STORED_DTYPE
            shape = tuple(int(s) for s in info["shape"])
            stored = adapter.map_tensor_name(name)
            n = int(np.prod(shape, dtype=np.int64)) if shape else 1
            self._weight_index.add(WeightEntry(stored, shape, dtype, data_nbytes=n * _WIDTH[dtype]))
            self._source[stored] = src
        adapter.sizes_of_tensors(self._config, {e.name: e.shape for e in self._weight_index})
        missing = [t for t in adapter.expected_tensors(self._config) if t not in self._weight_index] \
            if self._config.is_design else []
        if missing:
            raise ValueError(f"{path}: {len(missing)} tensors are missing, the first is '{missing[0]}'")
        self._tokenizer = None
        self._tokenizer_data = None

    @property
    def tokenizer(self):
        if self._tokenizer is None and os.path.exists(os.path.join(self._path, "tokenizer.json")):
            from .tokenizer import BPETokenizer
            self._tokenizer = BPETokenizer.from_hf_dir(self._path)
        return self._tokenizer

    def weight_data_section(self):
        raise ValueError("a model directory has no contiguous weight section")

    def view_data(self, entry: WeightEntry) -> np.ndarray:
        path, info, base = self._source[entry.name]
        raw = self._shards.view(path, info, base)
        if entry.dtype == "bfloat16":
            if info["dtype"] == "BF16":
                return np.frombuffer(raw, dtype=np.uint16).reshape(entry.shape)
            return round_bf16(_to_f32(raw, info["dtype"])).reshape(entry.shape)
        if entry.dtype == "int32":
            return np.frombuffer(raw, dtype=np.int32 if info["dtype"] == "I32" else np.int64).astype(
                np.int32).reshape(entry.shape)
        return _to_f32(raw, info["dtype"]).astype(np.float16).reshape(entry.shape)

    def get_weight_data(self, entry: WeightEntry) -> bytes:
        return self.view_data(entry).tobytes()

    def summary(self) -> str:
        c = self.config
        size = sum(os.path.getsize(p) for p in find_safetensor_files(self._path))
        return (f"model directory: {self._path}\n  {size:,} bytes of weights\n  arch {c.arch}: {c.num_layers} layers, "
                f"hidden {c.hidden_size}, heads {c.num_heads}/{c.num_kv_heads} x {c.head_dim}, intermediate "
                f"{c.intermediate_size}, vocab {c.vocab_size}, max_seq {c.max_seq_len}\n  tensors: "
                f"{len(self._weight_index)}")

    def close(self) -> None:
        shards = getattr(self, "_shards", None)
        if shards is not None:
            shards.close()


def open_model(path: str, int4_layout: Optional[str] = None) -> ZSELoader:
    """Loader of a ``.zse`` file or of a model directory."""
    if os.path.isdir(path):
        return DirectoryLoader(path)
    return ZSELoader(path, int4_layout=int4_layout)
