"""Pezarax: a decoder whose config.json lists its layers one by one, each with its mixer (`retention`, or `attention`:
differential attention in chunks) and an optional feed-forward of routed experts, which weight their input; plain pre-norms;
a stretch of layers that runs several times with the same weights and a memory of its own per pass, the embedding output
being added before every pass but the first.

Tensor names: `embed`, `head`, `final.norm`, and per layer `l<i>.norm1 / norm2`, `l<i>.mix.*`, `l<i>.mlp.router`,
`l<i>.mlp.e<j>.up / down`. The layers themselves are in `mixer_layers`, the step function in `runtime.mixer_runtime`.
"""
from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path

import torch

from . import mixer_checkpoint as mc
from . import mixer_layers as ml
from .mixer_checkpoint import load_tensors, save_checkpoint  # noqa: F401  (part of this module's interface)

ARCH = "Pezarax"

_MIXER_KEYS = {"retention": ("heads", "dim", "vdim", "decay"), "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "diff")}
MAX_EXPERTS, MAX_TOP = 512, 32


@dataclass
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None

    def __post_init__(self) -> None:
        if self.type not in _MIXER_KEYS:
            raise ValueError(f"unknown mixer {self.type!r}; known: {sorted(_MIXER_KEYS)}")
        m = self.mixer
        mc.require_keys(f"{self.type} layer", m, _MIXER_KEYS[self.type])
        rot = m.get("rot")
        if rot is not None and (rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"]):
            raise ValueError("an even number of rotated dimensions, at most the head's")
        if self.type == "retention":
            if len(m["decay"]) != m["heads"]:
                raise ValueError("one decay per head")
        else:
            if m["heads"] % m["kv_heads"]:
                raise ValueError("query heads are a multiple of the key/value heads")
            if (m.get("mask") or {}).get("size", 1) < 1:
                raise ValueError("a chunk holds at least one token")
        if self.mlp is not None:
            if self.mlp.get("kind", "moe") != "moe":
                raise ValueError(f"unknown feed-forward {self.mlp.get('kind')!r}")
            if not 1 <= self.experts <= MAX_EXPERTS or not 1 <= self.top <= min(self.experts, MAX_TOP):
                raise ValueError(f"routed experts: 1 to {MAX_EXPERTS}, of which a token uses 1 to {MAX_TOP}")

    @property
    def experts(self) -> int:
        return int(self.mlp["router"]["experts"])

    @property
    def top(self) -> int:
        return int(self.mlp["router"]["top"])

    @property
    def ff(self) -> int:
        return int(self.mlp["expert"]["ff"])


@dataclass
class PezaraxConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    logit_scale: float
    layers: list[LayerConfig]
    loop: tuple[int, int, int] | None = None      # first layer, first layer behind, passes

    def __post_init__(self) -> None:
        if self.loop is not None:
            a, b, n = self.loop
            if not 0 <= a <= b <= len(self.layers) or n < 1:
                raise ValueError(f"loop over layers {a} .. {b - 1}, {n} times: not within {len(self.layers)} layers")

    @classmethod
    def from_dict(cls, d: dict) -> "PezaraxConfig":
        mc.check_architecture(d, ARCH)
        lp = d.get("loop")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]), float(d["logit_scale"]),
                   [LayerConfig(L["type"], L["mixer"], L.get("mlp")) for L in d["layers"]],
                   (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None)

    @classmethod
    def load(cls, path: str | Path) -> "PezaraxConfig":
        return cls.from_dict(mc.read_config(path, ARCH))

    def to_dict(self) -> dict:
        d = {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "embedding": {"scale": self.embed_scale},
             "logit_scale": self.logit_scale, "layers": [{"type": L.type, "mixer": L.mixer, "mlp": L.mlp} for L in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d

    def passes(self) -> list[tuple[int, int]]:
        """(layer, pass) of every run of a layer, in order."""
        n = len(self.layers)
        a, b, times = self.loop or (0, 0, 1)
        return [(i, 0) for i in range(a)] + [(i, k) for k in range(times) for i in range(a, b)] + [(i, 0) for i in range(b, n)]


def tensor_plan(c: PezaraxConfig) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor."""
    W = c.width
    out: dict[str, tuple[int, ...]] = {"embed": (c.vocab, W), "final.norm": (W,), "head": (c.vocab, W)}
    for i, L in enumerate(c.layers):
        p, m = f"l{i}.", L.mixer
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if L.type == "retention":
            mix = {"q": (H * D, W), "k": (H * D, W), "v": (H * V, W), "g": (H * V, W)}
        else:
            G = m["kv_heads"]
            mix = {"q": (H * 2 * D, W), "k": (G * 2 * D, W), "v": (G * V, W), "lq1": (D,), "lk1": (D,), "lq2": (D,), "lk2": (D,)}
        mix["o"] = (W, H * V)
        out.update({p + "mix." + n: s for n, s in mix.items()})
        out[p + "norm1"] = (W,)
        if L.mlp is not None:
            out[p + "norm2"] = (W,)
            out[p + "mlp.router"] = (L.experts, W)
            for e in range(L.experts):
                out[p + f"mlp.e{e}.up"], out[p + f"mlp.e{e}.down"] = (L.ff, W), (W, L.ff)
    return out


def random_tensors(c: PezaraxConfig, seed: int = 0, device: str = "cpu", gain: float = 1.0) -> dict[str, torch.Tensor]:
    """Random weights of the design (bf16). `gain` scales the query and key projections."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_plan(c).items():
        base = name.rsplit(".mix.", 1)[-1]
        z = torch.randn(*shape, generator=g, device=device)
        if base in ("lq1", "lk1", "lq2", "lk2"):
            t = z * 0.6 * shape[0] ** -0.25
        elif len(shape) == 1:
            t = 1.0 + 0.1 * z
        elif name == "embed":
            t = z / c.embed_scale
        else:
            t = z * shape[1] ** -0.5 * (gain if base in ("q", "k") else 1.5 if name.endswith((".up", ".down")) else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def build_model(c: PezaraxConfig, tensors: dict[str, torch.Tensor], *, dtype: torch.dtype = torch.bfloat16, device: str = "cuda",
                slots: int = 8, pages: int = 64) -> ml.MixerModel:
    """Weights in the kernels' layout, with room for `slots` requests and `pages` pages of their positions."""
    mc.check_dtype(dtype)
    mc.check_tensors(tensor_plan(c), tensors)
    f32 = lambda n: tensors[n].float().to(device)
    layers = []
    for i, L in enumerate(c.layers):
        p = f"l{i}."
        w = {n[len(p) + 4:]: t for n, t in tensors.items() if n.startswith(p + "mix.")}
        if L.type == "retention":
            mixer = ml.RetentionMixer(w, L.mixer, c.eps, dtype, device, slots)
        else:
            mixer = ml.GroupedAttentionMixer(w, L.mixer, c.eps, dtype, device, pages, pages * ml.mo.PAGE, mask="chunk")
        layer = ml.MixerLayer(mixer, f32(p + "norm1"))
        if L.mlp is not None:
            q = p + "mlp."
            layer.mlp = ml.RoutedExperts(tensors[q + "router"], [tensors[q + f"e{e}.up"] for e in range(L.experts)],
                                         [tensors[q + f"e{e}.down"] for e in range(L.experts)], ml.mo.Router(L.experts, L.top), dtype, device)
            layer.norm2 = f32(p + "norm2")
        layers.append(layer)
    start = c.loop[0] if c.loop else 0
    runs = [layers[i] if k == 0 else layers[i].again(reinject=i == start) for i, k in c.passes()]
    return ml.MixerModel(c.vocab, c.width, c.eps, dtype, tensors["embed"].to(torch.bfloat16).contiguous().to(device), runs,
                         f32("final.norm") * c.logit_scale, ml.FusedLinear([("head", tensors["head"])], dtype, device), plus_one=False,
                         embed_scale=c.embed_scale)


def build_runtime(path, **kw):
    """Runtime over a checkpoint folder (see `mixer_checkpoint.open_runtime`)."""
    return mc.open_runtime(path, PezaraxConfig.load, build_model, **kw)
