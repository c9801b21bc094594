"""Zemozen: a decoder whose config.json lists its layers one by one, each with its mixer and an optional feed-forward of routed
experts, on plain pre-norms and a residual stream that takes every sublayer's output times a constant. Mixers:
  * `attention`: grouped-query attention in a window, norms and rotation (slowed down linearly) of queries and keys, values mixed
    with those of the first mixing layer, a sigmoid gate per head
  * `parallel`: attention in a window (rotated neighbours, capped scores, a sink of score 0) beside a Mamba-2 recurrence
The experts are SwiGLUs, the last ones of a router's outputs identities; a correction per expert counts for the choice alone.

Tensor names: `embed`, `head`, `final.norm`, and per layer `l<i>.norm1 / norm2`, `l<i>.mix.*` (`parallel`: `l<i>.mix.left.*` and
`l<i>.mix.right.*`), `l<i>.mlp.router / correction`, `l<i>.mlp.e<j>.gate / up / down`. The layers themselves are in
`mixer_layers`, the step function in `runtime.mixer_runtime`.
"""
from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path

import torch

from . import mixer_checkpoint as mc
from . import mixer_layers as ml
from .mixer_checkpoint import load_tensors, save_checkpoint  # noqa: F401  (part of this module's interface)

ARCH = "Zemozen"

_ATTENTION = ("heads", "kv_heads", "dim", "vdim", "scale")
_STATE_SPACE = ("heads", "vdim", "state", "groups", "conv", "norm_groups")
MAX_EXPERTS, MAX_TOP = 512, 32


def _check_attention(what: str, m: dict, keys=_ATTENTION) -> None:
    mc.require_keys(what, m, keys)
    rot = m.get("rot")
    if rot is not None and (rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"]):
        raise ValueError("an even number of rotated dimensions, at most the head's")
    if rot is not None and (rot.get("scaling") or {}).get("factor", 1.0) <= 0:
        raise ValueError("a positive factor slows rotations down")
    if m["heads"] % m["kv_heads"]:
        raise ValueError("query heads are a multiple of the key/value heads")
    if (m.get("mask") or {}).get("size", 1) < 1:
        raise ValueError("a window holds at least one token")


@dataclass
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None

    def __post_init__(self) -> None:
        m = self.mixer
        if self.type == "attention":
            _check_attention("attention layer", m)
        elif self.type == "parallel":
            mc.require_keys("parallel layer", m, ("left", "right", "left_scale", "right_scale"))
            _check_attention("left side", m["left"], _ATTENTION + ("softcap",))
            if not m["left"]["softcap"] > 0:
                raise ValueError("scores are capped at a positive value")
            r = m["right"]
            mc.require_keys("right side", r, _STATE_SPACE)
            if r["heads"] % r["groups"] or r["heads"] * r["vdim"] % r["norm_groups"] or r["conv"] < 1:
                raise ValueError("state space: heads a multiple of the groups, equal parts of the norm, at least one tap")
        else:
            raise ValueError(f"unknown mixer {self.type!r}; known: attention, parallel")
        if self.mlp is not None:
            if self.mlp.get("kind", "moe") != "moe":
                raise ValueError(f"unknown feed-forward {self.mlp.get('kind')!r}")
            n = self.experts + self.identity
            if self.experts < 1 or self.identity < 0 or n > MAX_EXPERTS or not 1 <= self.top <= min(n, MAX_TOP):
                raise ValueError(f"routed experts: up to {MAX_EXPERTS} with the identities, of which a token uses 1 to {MAX_TOP}")

    @property
    def experts(self) -> int:
        return int(self.mlp["router"]["experts"])

    @property
    def identity(self) -> int:
        return int(self.mlp["router"].get("identity") or 0)

    @property
    def top(self) -> int:
        return int(self.mlp["router"]["top"])

    @property
    def ff(self) -> int:
        return int(self.mlp["expert"]["ff"])

    @property
    def v_mix(self) -> bool:
        return self.type == "attention" and bool(self.mixer.get("v_mix"))


@dataclass
class ZemozenConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    residual_mult: float
    layers: list[LayerConfig]

    def __post_init__(self) -> None:
        if len({(L.mixer["kv_heads"], L.mixer["vdim"]) for L in self.layers if L.v_mix}) > 1:
            raise ValueError("layers that mix values have equal key/value heads and value sizes")

    @classmethod
    def from_dict(cls, d: dict) -> "ZemozenConfig":
        mc.check_architecture(d, ARCH)
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]), float(d["residual_mult"]),
                   [LayerConfig(L["type"], L["mixer"], L.get("mlp")) for L in d["layers"]])

    @classmethod
    def load(cls, path: str | Path) -> "ZemozenConfig":
        return cls.from_dict(mc.read_config(path, ARCH))

    def to_dict(self) -> dict:
        return {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "embedding": {"scale": self.embed_scale},
                "residual_mult": self.residual_mult, "layers": [{"type": L.type, "mixer": L.mixer, "mlp": L.mlp} for L in self.layers]}

    def first_v_mix(self) -> int:
        """The layer whose values later ones mix in (-1: there is none)."""
        return next((i for i, L in enumerate(self.layers) if L.v_mix), -1)


def _attention_plan(m: dict, width: int) -> dict[str, tuple[int, ...]]:
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": (H * D, width), "k": (G * D, width), "v": (G * V, width), "q.norm": (D,), "k.norm": (D,), "o": (width, H * V)}


def tensor_plan(c: ZemozenConfig) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor."""
    W = c.width
    out: dict[str, tuple[int, ...]] = {"embed": (c.vocab, W), "final.norm": (W,), "head": (c.vocab, W)}
    for i, L in enumerate(c.layers):
        p, m = f"l{i}.", L.mixer
        if L.type == "attention":
            mix = _attention_plan(m, W) | {"g": (m["heads"], W)}
            if L.v_mix:
                mix["vmix"] = ()
        else:
            r = m["right"]
            H, inner = r["heads"], r["heads"] * r["vdim"]
            ch = inner + 2 * r["groups"] * r["state"]
            mix = {"left." + n: s for n, s in _attention_plan(m["left"], W).items()}
            mix.update({"right." + n: s for n, s in {"in": (inner + ch + H, W), "conv": (ch, r["conv"]), "conv.b": (ch,), "dt_bias": (H,), "A_log": (H,),
                                                     "D": (H,), "norm": (inner,), "o": (W, inner)}.items()})
        out.update({p + "mix." + n: s for n, s in mix.items()})
        out[p + "norm1"] = (W,)
        if L.mlp is not None:
            n = L.experts + L.identity
            out.update({p + "norm2": (W,), p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
            for e in range(L.experts):
                q = p + f"mlp.e{e}."
                out[q + "gate"], out[q + "up"], out[q + "down"] = (L.ff, W), (L.ff, W), (W, L.ff)
    return out


def random_tensors(c: ZemozenConfig, seed: int = 0, device: str = "cpu", gain: float = 1.0) -> dict[str, torch.Tensor]:
    """Random weights of the design (bf16). `gain` scales the norms of queries and keys."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_plan(c).items():
        base = name.rsplit(".", 1)[-1]
        z = torch.randn(shape, generator=g, device=device)
        if base == "vmix":
            t = 0.4 + 0.1 * z
        elif base == "A_log":
            t = 0.5 + 0.8 * z
        elif base == "dt_bias":
            t = z - 2.5
        elif name.endswith("conv.b"):
            t = 0.2 * z
        elif base == "correction":
            t = 0.1 * z
        elif name.endswith((".q.norm", ".k.norm")):
            t = gain * (1.0 + 0.1 * z)
        elif len(shape) == 1:
            t = 1.0 + 0.1 * z
        elif base == "embed":
            t = z / c.embed_scale
        else:
            t = z * shape[1] ** -0.5 * (1.5 if base in ("gate", "up", "down") else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def build_model(c: ZemozenConfig, tensors: dict[str, torch.Tensor], *, dtype: torch.dtype = torch.bfloat16, device: str = "cuda",
                slots: int = 8, pages: int = 64) -> ml.MixerModel:
    """Weights in the kernels' layout, with room for `slots` requests and `pages` pages of their positions."""
    mc.check_dtype(dtype)
    mc.check_tensors(tensor_plan(c), tensors)
    f32 = lambda n: tensors[n].float().to(device)
    sub = lambda p: {n[len(p):]: t for n, t in tensors.items() if n.startswith(p)}
    context, first = pages * ml.mo.PAGE, c.first_v_mix()
    layers = []
    for i, L in enumerate(c.layers):
        p, m = f"l{i}.", L.mixer
        if L.type == "attention":
            mixer = ml.GroupedAttentionMixer(sub(p + "mix."), m, c.eps, dtype, device, pages, context,
                                             v_mix=None if not L.v_mix else "first" if i == first else "mix")
        else:
            wl, wr = sub(p + "mix.left."), sub(p + "mix.right.")
            left = ml.GroupedAttention(wl, m["left"], c.eps, dtype, device, pages, context, neighbours=True, sink=0.0, scale_out=float(m["left_scale"]))
            right = ml.StateSpaceMixer(wr, m["right"], c.eps, dtype, device, slots, scale=float(m["right_scale"]))
            mixer = ml.ParallelMixer(left, right, wl, wr, dtype, device)
        layer = ml.MixerLayer(mixer, f32(p + "norm1"))
        if L.mlp is not None:
            q = p + "mlp."
            up, down, gate = ([tensors[q + f"e{e}.{n}"] for e in range(L.experts)] for n in ("up", "down", "gate"))
            router = ml.mo.Router(L.experts, L.top, score="softmax", renorm=True, on_output=True, identity=L.identity)
            layer.mlp = ml.RoutedExperts(tensors[q + "router"], up, down, router, dtype, device, gate=gate, correction=tensors[q + "correction"])
            layer.norm2 = f32(p + "norm2")
        layers.append(layer)
    return ml.MixerModel(c.vocab, c.width, c.eps, dtype, tensors["embed"].to(torch.bfloat16).contiguous().to(device), layers, f32("final.norm"),
                         ml.FusedLinear([("head", tensors["head"])], dtype, device), plus_one=False, embed_scale=c.embed_scale,
                         residual_scale=c.residual_mult)


def build_runtime(path, **kw):
    """Runtime over a checkpoint folder (see `mixer_checkpoint.open_runtime`)."""
    return mc.open_runtime(path, ZemozenConfig.load, build_model, **kw)
