"""A checkpoint directory opened as if it were a GGUF file: metadata and tensors come from the converter, nothing is written."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import numpy as np

from ..gguf.reader import GGUFFile, TensorInfo
from ..gguf.writer import WriteTensor


@dataclass
class FolderGGUF(GGUFFile):
    arrays: dict[str, WriteTensor] = field(default_factory=dict, repr=False)

    def tensor_bytes(self, name: str) -> np.ndarray:
        d = self.arrays[name].data
        return np.asarray(d() if callable(d) else d).reshape(-1).view(np.uint8)

    def close(self) -> None:
        self.arrays = {}


def open_folder(path: str, outtype: str = "auto") -> FolderGGUF:
    """Open the checkpoint directory ``path`` (config.json + *.safetensors, tokenizer files where the architecture needs them)."""
    from .hf import checkpoint_parts
    with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
        cfg = json.load(f)
    kv, tensors = checkpoint_parts(path, cfg, outtype)
    arrays = {t.name: t for t in tensors}
    infos = {n: TensorInfo(n, tuple(t.shape), t.dtype, 0, t.nbytes) for n, t in arrays.items()}
    arch = kv["general.architecture"]
    full = {k if k.startswith(("general.", "tokenizer.", "adapter.", arch + ".")) else f"{arch}.{k}": v for k, v in kv.items()}
    return FolderGGUF(path, 3, "<", full, {}, infos, 0, 32, arrays=arrays)
