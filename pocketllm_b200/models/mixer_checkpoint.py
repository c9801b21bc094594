"""Checkpoint folders of decoders made of mixer layers: `config.json` (with `architecture`) and `model.safetensors`. What the
designs share: reading and writing the folder, checking names and shapes, opening a runtime with a pool of pages and slots."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Callable

import torch

from ..formats import safetensors_io as st_io
from ..ops import mixer_ops as mo


def read_config(path: str | Path, arch: str) -> dict:
    p = Path(path)
    return check_architecture(json.loads((p / "config.json" if p.is_dir() else p).read_text()), arch)


def check_architecture(d: dict, arch: str) -> dict:
    if d.get("architecture") != arch:
        raise ValueError(f"architecture {d.get('architecture')!r} is not {arch}")
    return d


def require_keys(what: str, d: dict, keys) -> None:
    missing = [k for k in keys if k not in d]
    if missing:
        raise ValueError(f"{what} without {missing}")


def save_checkpoint(directory: str | Path, config, tensors: dict[str, torch.Tensor]) -> None:
    d = Path(directory)
    d.mkdir(parents=True, exist_ok=True)
    (d / "config.json").write_text(json.dumps(config.to_dict()))
    st_io.write_file(d / "model.safetensors", tensors)


def load_tensors(path: str | Path) -> dict[str, torch.Tensor]:
    src = st_io.SafetensorsModel(path)
    return {n: src.get(n) for n in src.keys()}


def check_tensors(plan: dict[str, tuple[int, ...]], tensors: dict[str, torch.Tensor], free: tuple[str, ...] = ()) -> None:
    """Every planned tensor is there and has its shape (`free`: endings of matrices whose sizes only the tensors tell)."""
    for name, shape in plan.items():
        if name not in tensors:
            raise KeyError(f"missing tensor {name}")
        got = tuple(tensors[name].shape)
        if got != shape and not (name.endswith(free) and len(got) == len(shape) if free else False):
            raise ValueError(f"{name}: shape {got}, expected {shape}")


def check_dtype(dtype: torch.dtype) -> None:
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("dtype must be bfloat16 or float32")


def open_runtime(path, load_config: Callable, build_model: Callable, *, dtype: torch.dtype = torch.bfloat16, device: str = "cuda",
                 max_requests: int = 8, max_tokens: int | None = None, max_context: int = 4096, **kw):
    """Runtime over a checkpoint folder. `max_tokens`: positions that live requests hold at any time, all together (default:
    `max_context` for every slot)."""
    from ..runtime.mixer_runtime import MixerRuntime
    per = (max_context + mo.PAGE - 1) // mo.PAGE
    pages = max_requests * per if max_tokens is None else (max_tokens + mo.PAGE - 1) // mo.PAGE
    model = build_model(load_config(path), load_tensors(path), dtype=dtype, device=device, slots=max_requests, pages=pages)
    return MixerRuntime(model, max_requests=max_requests, pages=pages, device=device, **kw)
