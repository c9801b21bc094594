"""Gidisun: a decoder whose config.json lists its layers one by one, each with its mixer (`mlstm`, `gla` or
`latent_attention`), the mixer's sizes and an optional SwiGLU feed-forward; sandwich norms with weights stored around zero,
untied output matrix, no final cap.

Tensor names: `embed`, `head`, `final.norm`, and per layer `l<i>.norm1 / norm1b / norm2 / norm2b`, `l<i>.mix.*`, `l<i>.mlp.*`.
The layers themselves are in `mixer_layers`, the step function in `runtime.mixer_runtime`.
"""
from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path

import torch

from . import mixer_checkpoint as mc
from . import mixer_layers as ml
from .mixer_checkpoint import load_tensors, save_checkpoint  # noqa: F401  (part of this module's interface)

ARCH = "Gidisun"

# what a mixer's entry in the configuration has to name
_MIXER_KEYS = {"mlstm": ("heads", "dim", "vdim", "gate_cap"), "gla": ("heads", "dim", "vdim", "tau"),
               "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot")}


@dataclass
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None

    def __post_init__(self) -> None:
        if self.type not in _MIXER_KEYS:
            raise ValueError(f"unknown mixer {self.type!r}; known: {sorted(_MIXER_KEYS)}")
        mc.require_keys(f"{self.type} layer", self.mixer, _MIXER_KEYS[self.type])
        if self.mlp is not None and self.mlp.get("kind", "dense") != "dense":
            raise ValueError(f"unknown feed-forward {self.mlp.get('kind')!r}")
        if self.type == "latent_attention":
            m = self.mixer
            if m["rot"]["dims"] != m["rot_dim"] or m["rot_dim"] % 2:
                raise ValueError("latent attention rotates all of its (even) rotated part")
            if (m.get("mask") or {}).get("size", 1) < 1:
                raise ValueError("a window holds at least the token itself")


@dataclass
class GidisunConfig:
    vocab: int
    width: int
    eps: float
    layers: list[LayerConfig]

    @classmethod
    def from_dict(cls, d: dict) -> "GidisunConfig":
        mc.check_architecture(d, ARCH)
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]),
                   [LayerConfig(L["type"], L["mixer"], L.get("mlp")) for L in d["layers"]])

    @classmethod
    def load(cls, path: str | Path) -> "GidisunConfig":
        return cls.from_dict(mc.read_config(path, ARCH))

    def to_dict(self) -> dict:
        return {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "layers": [{"type": L.type, "mixer": L.mixer, "mlp": L.mlp} for L in self.layers]}


def tensor_plan(c: GidisunConfig, decay_rank: int = 16) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor. The rank of GLA's decay projection is not in the configuration (its tensors tell)."""
    W = c.width
    out: dict[str, tuple[int, ...]] = {"embed": (c.vocab, W), "final.norm": (W,), "head": (c.vocab, W)}
    for i, L in enumerate(c.layers):
        p, m = f"l{i}.", L.mixer
        H, D, V = m["heads"], m["dim"], m["vdim"]
        mix: dict[str, tuple[int, ...]] = {"o": (W, H * V)}
        if L.type == "latent_attention":
            R, K = m["rot_dim"], m["kv_rank"]
            mix.update({"q": (H * (D + R), W), "dkv": (K + R, W), "dkv.norm": (K,), "uk": (H * D, K), "uv": (H * V, K), "sink": (H,)})
        else:
            mix.update({"q": (H * D, W), "k": (H * D, W), "v": (H * V, W), "g": (H * V, W)})
            if L.type == "mlstm":
                mix.update({"i": (H, W), "i.b": (H,), "f": (H, W), "f.b": (H,), "norm": (H * V,)})
            else:
                mix.update({"a1": (decay_rank, W), "a2": (H * D, decay_rank), "a2.b": (H * D,), "norm": (V,)})
        out.update({p + "mix." + n: s for n, s in mix.items()})
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if L.mlp is not None:
            ff = L.mlp["ff"]
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_tensors(c: GidisunConfig, seed: int = 0, decay_rank: int = 16, device: str = "cpu", gain: float = 1.0) -> dict[str, torch.Tensor]:
    """Random weights of the design (bf16). `gain` scales the query and key projections."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_plan(c, decay_rank).items():
        base = name.rsplit(".mix.", 1)[-1]
        z = torch.randn(*shape, generator=g, device=device)
        if base == "f.b":
            t = 3.0 + z
        elif base == "a2.b":
            t = 2.0 + z
        elif base in ("i.b", "sink"):
            t = 0.5 * z
        elif base in ("norm", "dkv.norm"):
            t = 1.0 + 0.1 * z
        elif len(shape) == 1:
            t = 0.1 * z
        elif name == "embed":
            t = z
        else:
            t = z * shape[1] ** -0.5 * (gain if base in ("q", "k", "uk") else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def build_model(c: GidisunConfig, tensors: dict[str, torch.Tensor], *, dtype: torch.dtype = torch.bfloat16, device: str = "cuda",
                slots: int = 8, pages: int = 64) -> ml.MixerModel:
    """Weights in the kernels' layout, with room for `slots` requests and `pages` pages of their positions."""
    mc.check_dtype(dtype)
    mc.check_tensors(tensor_plan(c), tensors, free=("mix.a1", "mix.a2"))
    f32 = lambda n: tensors[n].float().to(device)
    layers = []
    for i, L in enumerate(c.layers):
        p = f"l{i}."
        w = {n[len(p) + 4:]: t for n, t in tensors.items() if n.startswith(p + "mix.")}
        if L.type in ml.PAGED:
            mixer = ml.MIXERS[L.type](w, L.mixer, c.eps, dtype, device, pages, pages * ml.mo.PAGE)
        else:
            mixer = ml.MIXERS[L.type](w, L.mixer, c.eps, dtype, device, slots)
        layer = ml.MixerLayer(mixer, f32(p + "norm1"), norm1b=f32(p + "norm1b"))
        if L.mlp is not None:
            layer.mlp = ml.SwiGLU({n: tensors[p + "mlp." + n] for n in ("gate", "up", "down")}, dtype, device)
            layer.norm2, layer.norm2b = f32(p + "norm2"), f32(p + "norm2b")
        layers.append(layer)
    return ml.MixerModel(c.vocab, c.width, c.eps, dtype, tensors["embed"].to(torch.bfloat16).contiguous().to(device), layers, f32("final.norm"),
                         ml.FusedLinear([("head", tensors["head"])], dtype, device))


def build_runtime(path, **kw):
    """Runtime over a checkpoint folder (see `mixer_checkpoint.open_runtime`)."""
    return mc.open_runtime(path, GidisunConfig.load, build_model, **kw)
