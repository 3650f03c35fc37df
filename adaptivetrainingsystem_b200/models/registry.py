"""Model classes by the name in a model folder's ``config.json`` (``architecture``), and loading of such a folder.

A model folder holds ``config.json`` and ``model.safetensors``.  Without an ``architecture`` key the folder is taken for a
:class:`DeepSeekTransformer` whose configuration has the fields of :class:`ModelConfig`.
"""
from __future__ import annotations

import json
import os
import struct
from dataclasses import dataclass
from typing import Any, Callable, Dict, Iterator, Tuple, Type

import torch

from ..config import ModelConfig, NemipelConfig, VimodraConfig
from .layered import LayeredDecoder
from .nemipel import Nemipel
from .transformer import DeepSeekTransformer
from .vimodra import Vimodra

_DTYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I64": torch.int64, "I32": torch.int32, "I16": torch.int16,
           "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


class SafetensorsFile:
    """Reads one tensor at a time: eight bytes of header length (little endian), the JSON header, the data."""

    def __init__(self, path: str):
        self.path = path
        with open(path, "rb") as f:
            (n,) = struct.unpack("<Q", f.read(8))
            if n > os.path.getsize(path) - 8:
                raise ValueError(f"{path}: the header does not fit the file")
            self.header: Dict[str, Dict[str, Any]] = json.loads(f.read(n))
        self.header.pop("__metadata__", None)
        self.start = 8 + n

    def keys(self) -> Iterator[str]:
        return iter(self.header)

    def tensor(self, name: str) -> torch.Tensor:
        e = self.header[name]
        a, b = e["data_offsets"]
        with open(self.path, "rb") as f:
            f.seek(self.start + a)
            raw = bytearray(f.read(b - a))
        if len(raw) != b - a:
            raise ValueError(f"{self.path}: {name} is cut off")
        dtype = _DTYPES[e["dtype"]]
        return torch.frombuffer(raw, dtype=dtype).reshape(e["shape"]) if raw else torch.empty(e["shape"], dtype=dtype)


@dataclass(frozen=True)
class ModelEntry:
    config: Callable[[Dict[str, Any]], Any]                              # config.json -> configuration
    load: Callable[[Any, SafetensorsFile, torch.dtype, torch.device], Any]
    cls: type


def _load_deepseek(cfg: ModelConfig, file: SafetensorsFile, dtype, device):
    cfg.gradient_checkpointing = False
    model = DeepSeekTransformer(cfg)
    model.load_state_dict({k: file.tensor(k) for k in file.keys()}, strict=False)
    return model.to(device, dtype).eval()


def _layered(config: Callable[[Dict[str, Any]], Any], cls: Type[LayeredDecoder]) -> ModelEntry:
    return ModelEntry(config, lambda cfg, file, dtype, device: cls.from_tensors(cfg, file.tensor, list(file.keys()), dtype, device), cls)


MODELS: Dict[str, ModelEntry] = {
    "DeepSeekTransformer": ModelEntry(ModelConfig.from_dict, _load_deepseek, DeepSeekTransformer),
    "Vimodra": _layered(VimodraConfig.from_dict, Vimodra),
    "Nemipel": _layered(NemipelConfig.from_dict, Nemipel),
}


def register_model(name: str, entry: ModelEntry) -> None:
    MODELS[name] = entry


def read_config(folder: str) -> Tuple[ModelEntry, Any]:
    with open(os.path.join(folder, "config.json")) as f:
        d = json.load(f)
    name = d.get("architecture", "DeepSeekTransformer")
    if name not in MODELS:
        raise ValueError(f"{folder}: unknown architecture {name!r} (known: {sorted(MODELS)})")
    return MODELS[name], MODELS[name].config(d)


def load_model(folder: str, dtype: torch.dtype = torch.bfloat16, device="cuda"):
    """The model of a folder, in inference mode."""
    entry, cfg = read_config(folder)
    return entry.load(cfg, SafetensorsFile(os.path.join(folder, "model.safetensors")), dtype, torch.device(device))
