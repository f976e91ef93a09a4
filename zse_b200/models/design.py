"""What the models share whose config.json describes every layer on its own: number formats, weights, typed buffers."""
from __future__ import annotations

from typing import Optional

import numpy as np
import torch

from ..format.loader import ZSELoader
from .decoder import DecoderModel

SHORT_CHUNK = 16            # chunks up to this length run token by token
PLANE_ROWS = 256            # passes up to this size take projections as fp32 split-K planes


class WeightReader:
    """Tensors of a model at the width the model runs in, copied out of the file (or its streamed device mirror)."""

    def __init__(self, model: "DesignModel", loader: ZSELoader):
        self.model, self.loader, self.mirror = model, loader, None
        self.act, self.dev = model.act_dtype, model.device
        if self.dev.type == "cuda":
            from ..runtime.weight_stream import open_mirror
            self.mirror = open_mirror(loader, self.dev, model.load_stats)

    def tensor(self, name: str) -> torch.Tensor:
        e = self.loader.weight_index.find(name)
        if e is None:
            raise KeyError(name)
        if self.mirror is not None:
            t = self.mirror.view(e.data_offset, e.data_nbytes, e.dtype).reshape(e.shape)
        else:
            a = np.array(self.loader.view_data(e))
            t = torch.from_numpy(a.view(np.int16)).view(torch.bfloat16) if e.dtype == "bfloat16" else torch.from_numpy(a)
            t = t.to(self.dev)
        return t.to(self.act)

    def keep(self, t: torch.Tensor) -> torch.Tensor:
        """A copy of its own (a mirror's views go away with it)."""
        t = self.model.ops.dense(t.clone(memory_format=torch.contiguous_format), self.act)
        self.model.weight_bytes += t.numel() * t.element_size()
        return t

    def get(self, name: str) -> torch.Tensor:
        return self.keep(self.tensor(name))

    def linear(self, name: str):
        return self.model.ops.dense_linear(self.get(name))

    def stack(self, parts, rows: int, width: int) -> torch.Tensor:
        """``parts``: (first row, tensor); rows between them are zero."""
        out = torch.zeros(rows, width, dtype=self.act, device=self.dev)
        for at, t in parts:
            out[at: at + t.shape[0]] = t
        return self.keep(out)

    def release(self) -> None:
        if self.mirror is not None:
            self.mirror.release()


class DesignModel(DecoderModel):
    act_dtype = torch.bfloat16
    mixed_passes = True

    def set_dtype(self, dtype: Optional[str]) -> None:
        kinds = {None: torch.bfloat16, "bfloat16": torch.bfloat16, "float32": torch.float32}
        if dtype not in kinds:
            raise ValueError(f"'{self.config.arch}' runs in bfloat16 or float32, not {dtype}")
        self.act_dtype = kinds[dtype]

    def _open(self, loader: ZSELoader) -> WeightReader:
        if self.plan.tp_size != 1:
            raise NotImplementedError(f"'{self.config.arch}' is served by one GPU (no tensor-parallel split of its layers "
                                      f"yet)")
        self.cache_block_size = 64
        return WeightReader(self, loader)
