"""In-memory checkpoint: tensors kept as raw GGUF block bytes + type + logical shape.

``ModelWeights`` is what both the torch reference model (after dequantisation) and the GPU
engine (after the load-time tile reorder) are built from.  It can come from a ``.gguf`` file
or from the synthetic generator, and can be written back to a ``.gguf``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Mapping

import torch

from ..gguf import GGMLType, GGUFFile, GGUFWriter, dequantize, quantize
from ..gguf.constants import BLOCK_GEOMETRY
from .config import ModelConfig


@dataclass
class QTensor:
    qtype: GGMLType
    shape: tuple[int, ...]          # logical shape, torch order
    raw: torch.Tensor               # flat uint8

    def to_float(self) -> torch.Tensor:
        return dequantize(self.raw, self.qtype, self.shape)

    @property
    def row_bytes(self) -> int:
        e, b = BLOCK_GEOMETRY[self.qtype]
        return self.shape[-1] // e * b

    def rows(self, start: int, stop: int) -> "QTensor":
        """Row slice of a 2-D tensor (column-parallel / vocab-parallel shards)."""
        assert len(self.shape) == 2
        rb = self.row_bytes
        return QTensor(self.qtype, (stop - start, self.shape[1]), self.raw[start * rb:stop * rb])

    def cols(self, start: int, stop: int) -> "QTensor":
        """Column slice of a 2-D tensor on block boundaries (row-parallel shards)."""
        assert len(self.shape) == 2
        e, b = BLOCK_GEOMETRY[self.qtype]
        if start % e or stop % e:
            raise ValueError(f"column slice [{start},{stop}) is not aligned to {self.qtype.name} blocks of {e}")
        r = self.raw.reshape(self.shape[0], self.row_bytes)
        return QTensor(self.qtype, (self.shape[0], stop - start),
                       r[:, start // e * b: stop // e * b].contiguous().reshape(-1))

    def expert(self, e: int) -> "QTensor":
        assert len(self.shape) == 3
        n = self.raw.numel() // self.shape[0]
        return QTensor(self.qtype, self.shape[1:], self.raw[e * n:(e + 1) * n])

    def to(self, device) -> "QTensor":
        return QTensor(self.qtype, self.shape, self.raw.to(device))

    def transcoded(self, target: GGMLType = GGMLType.Q8_0) -> "QTensor":
        """The same values re-encoded in ``target`` (decode, then quantise; one leading slice at a time so that the fp32
        temporary stays small).  Used where a kernel needs a format with a packed device layout and the file's format has
        none: Q8_0 adds a rounding error of ~0.4 %, far below the error of the 1- to 3-bit formats it replaces."""
        if self.qtype == target:
            return self
        if len(self.shape) < 3:
            return QTensor(target, self.shape, quantize(self.to_float(), target))
        parts = [self.expert(e).transcoded(target).raw for e in range(self.shape[0])]
        return QTensor(target, self.shape, torch.cat(parts))


class ModelWeights:
    def __init__(self, config: ModelConfig, tensors: dict[str, QTensor], metadata: dict | None = None):
        self.config = config
        self.tensors = tensors
        self.metadata = metadata or {}

    def __getitem__(self, name: str) -> QTensor:
        return self.tensors[name]

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def get(self, name: str):
        return self.tensors.get(name)

    def float_dict(self, device="cpu") -> dict[str, torch.Tensor]:
        """Every tensor dequantised to float32 (only sensible for small models)."""
        return {k: dequantize(v.raw.to(device), v.qtype, v.shape) for k, v in self.tensors.items()}

    def nbytes(self) -> int:
        return sum(t.raw.numel() for t in self.tensors.values())

    # -- file I/O ------------------------------------------------------------------------------
    @staticmethod
    def from_path(path: str, device="cpu") -> "ModelWeights":
        """A `.gguf` file, or a checkpoint directory of a family that is served without conversion."""
        return ModelWeights.from_directory(path) if os.path.isdir(path) else ModelWeights.from_gguf(path, device)

    @staticmethod
    def from_directory(path: str) -> "ModelWeights":
        """`config.json` + `*.safetensors`; the family's reader is chosen by the configuration's "architecture"."""
        from .convert_hf import load_checkpoint, tokenizer_metadata
        with open(os.path.join(path, "config.json")) as f:
            arch = json.load(f).get("architecture")
        reader = _directory_readers().get(arch)
        if reader is None:
            raise ValueError(f"{path}: no reader for architecture {arch!r} (known: {', '.join(_directory_readers())}; "
                             "Hugging Face checkpoints are converted to GGUF first: python -m llaminar_b200.models.convert_hf)")
        w = reader(*load_checkpoint(path))
        if os.path.exists(os.path.join(path, "tokenizer.json")):
            w.metadata.update(tokenizer_metadata(path))
        return w

    @staticmethod
    def from_gguf(path: str, device="cpu") -> "ModelWeights":
        gf = GGUFFile(path)
        cfg = ModelConfig.from_gguf(gf)
        tensors = {}
        for t in gf:
            raw = t.raw()
            raw = raw.to(device) if str(device) != "cpu" else raw.clone()
            tensors[t.name] = QTensor(t.qtype, t.shape, raw)
        md = dict(gf.metadata)
        gf.close()
        return ModelWeights(cfg, tensors, md)

    def save_gguf(self, path: str, extra_metadata: dict | None = None) -> None:
        w = GGUFWriter()
        md = dict(self.config.gguf_metadata())
        for k, v in self.metadata.items():
            if k != "general.alignment":
                md.setdefault(k, v)
        md.update(extra_metadata or {})
        for k, v in md.items():
            w.add(k, v)
        for name, t in self.tensors.items():
            w.add_raw_tensor(name, t.qtype, t.shape, t.raw)
        w.write(path)


def _directory_readers() -> dict:
    """config.json "architecture" -> function(config dict, {name: tensor}) -> ModelWeights."""
    from . import kefasun, lagedra, pozivik, zogepel
    return {m.ARCHITECTURE: m.weights_from_tensors for m in (kefasun, lagedra, pozivik, zogepel)}


def qtensor_from_float(x: torch.Tensor, qtype: GGMLType) -> QTensor:
    return QTensor(GGMLType(qtype), tuple(x.shape), quantize(x, qtype))


def named_weights(cfg: ModelConfig, names: list[tuple[str, str, str, tuple[int, ...]]], tensors: Mapping[str, torch.Tensor]) -> ModelWeights:
    """A checkpoint's tensors under the package's names.  ``names``: (checkpoint name, package name, kind, shape), kind "mat" a
    matrix, "vec" a vector kept as it is, "taps" small filters [channels, taps] kept likewise, "num" a single number (a vector of
    one), "gain" a zero-centred norm gain (stored as 1 + w), "stack" matrices of the names that "{}" in ``src`` stands for (0, 1,
    ...), one behind the other."""
    out: dict[str, QTensor] = {}

    def take(src: str, shape: tuple[int, ...]) -> torch.Tensor:
        if src not in tensors:
            raise KeyError(f"tensor '{src}' is missing from the checkpoint")
        x = tensors[src]
        if tuple(x.shape) != shape:
            raise ValueError(f"tensor '{src}' has shape {tuple(x.shape)}, the configuration says {shape}")
        return x

    for src, dst, kind, shape in names:
        x = torch.stack([take(src.format(i), shape[1:]) for i in range(shape[0])]) if kind == "stack" else take(src, () if kind == "num" else shape).reshape(shape)
        if kind in ("mat", "stack"):
            out[dst] = qtensor_from_float(x.float().contiguous(), GGMLType.F32 if x.dtype == torch.float32 else GGMLType.BF16)
        else:
            out[dst] = qtensor_from_float((1.0 + x.float() if kind == "gain" else x.float()).contiguous(), GGMLType.F32)
    return ModelWeights(cfg, out, {})
