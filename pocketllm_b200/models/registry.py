"""Architecture registry: what a checkpoint says it is -> model runtime builder. GGUF files name their architecture in
`general.architecture`, Safetensors folders in config.json (`architecture`)
(reference: src/components/moe/registry.py `detect_spec`)."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Callable

_BUILDERS: dict[str, Callable] = {}
_FOLDERS: set[str] = set()      # architectures whose checkpoints are Safetensors folders


def register(arch: str, folder: bool = False):
    def deco(fn):
        _BUILDERS[arch] = fn
        if folder:
            _FOLDERS.add(arch)
        return fn
    return deco


def architectures() -> list[str]:
    _load()
    return sorted(_BUILDERS)


def folder_architecture(path) -> str | None:
    """The registered architecture of a Safetensors folder, or None when its config.json names no registered one."""
    _load()
    f = Path(path) / "config.json"
    if not f.is_file():
        return None
    arch = json.loads(f.read_text()).get("architecture")
    return arch if arch in _FOLDERS else None


def build_runtime(path, architecture: str | None = None, **kw):
    """Open `path`, pick the builder for its architecture and return a token runtime."""
    from ..formats import gguf
    _load()
    if architecture is None and Path(path).is_dir() and (Path(path) / "config.json").is_file():
        architecture = json.loads((Path(path) / "config.json").read_text()).get("architecture")
        if architecture not in _FOLDERS:
            raise KeyError(f"no runtime for architecture {architecture!r}; known: {sorted(_FOLDERS)}")
    arch = architecture or gguf.GGUFFile(gguf.shard_paths(path)[0]).architecture()
    if arch not in _BUILDERS:
        raise KeyError(f"no runtime for GGUF architecture {arch!r}; known: {sorted(_BUILDERS)}")
    return _BUILDERS[arch](path, **kw)


def _load() -> None:
    if _BUILDERS:
        return

    @register("minimax-m2")
    def _mm(path, **kw):
        from . import minimax_m2
        return minimax_m2.MiniMaxM2Model(path, **kw)

    @register("glm-dsa")
    def _glm(path, **kw):
        from . import glm_dsa
        return glm_dsa.GLMDSAModel(path, **kw)

    @register("Gidisun", folder=True)
    def _gidisun(path, **kw):
        from . import gidisun
        return gidisun.build_runtime(path, **kw)

    @register("Pezarax", folder=True)
    def _pezarax(path, **kw):
        from . import pezarax
        return pezarax.build_runtime(path, **kw)

    @register("Zemozen", folder=True)
    def _zemozen(path, **kw):
        from . import zemozen
        return zemozen.build_runtime(path, **kw)

    @register("Zarinex", folder=True)
    def _zarinex(path, **kw):
        from . import zarinex
        return zarinex.build_runtime(path, **kw)
