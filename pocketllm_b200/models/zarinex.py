"""Zarinex: a decoder whose config.json lists its layers one by one, each with its mixer and an optional feed-forward of routed experts
beside a shared one. Norms follow the sums, x <- norm(alpha x + gate * sublayer(x)), with a sigmoid gate per element on every sublayer's
result; every mixer reads a mix of its input with the previous token's; a sinusoid of the position is added to the embedding, whose
table is also the output matrix. A layer may use another layer's weights with a state or cache of its own (`weights_of`). Mixers:
  * `mamba1`: selective scan, a decay per channel and state
  * `latent_attention`: queries, keys and values from latents, no positions, a gate on the heads' outputs
  * `hgrn2`: linear attention whose forget gate also decides what is written

Tensor names: `embed`, `final.norm`, and per layer with weights of its own `l<i>.norm1 / norm2`, `l<i>.shift`, `l<i>.rg1 / rg1.b / rg2 /
rg2.b`, `l<i>.mix.*`, `l<i>.mlp.router / router.b`, `l<i>.mlp.e<j>.* / shared.*` with `gate / up / down`. The layers themselves are in
`mixer_layers`, the step function in `runtime.mixer_runtime`.
"""
from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path

import torch

from . import mixer_checkpoint as mc
from . import mixer_layers as ml
from .mixer_checkpoint import load_tensors, save_checkpoint  # noqa: F401  (part of this module's interface)

ARCH = "Zarinex"

_MIXER_KEYS = {"mamba1": ("inner", "state", "dt_rank", "conv"), "latent_attention": ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale"),
               "hgrn2": ("heads", "dim", "vdim")}
MAX_EXPERTS, MAX_TOP = 512, 32


@dataclass
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None
    weights_of: int | None = None

    def __post_init__(self) -> None:
        if self.type not in _MIXER_KEYS:
            raise ValueError(f"unknown mixer {self.type!r}; known: {sorted(_MIXER_KEYS)}")
        m = self.mixer
        mc.require_keys(f"{self.type} layer", m, _MIXER_KEYS[self.type])
        if any(m[k] < 1 for k in _MIXER_KEYS[self.type] if k != "scale"):
            raise ValueError(f"{self.type} layer: sizes are at least one")
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

    @property
    def shared_ff(self) -> int:
        """Hidden size of the shared expert (0: there is none)."""
        return int((self.mlp.get("shared") or {}).get("ff") or 0)

    def to_dict(self) -> dict:
        d = {"type": self.type, "mixer": self.mixer, "mlp": self.mlp}
        return d if self.weights_of is None else d | {"weights_of": self.weights_of}


@dataclass
class ZarinexConfig:
    vocab: int
    width: int
    eps: float
    alpha: float
    layers: list[LayerConfig]

    def __post_init__(self) -> None:
        if not self.layers:
            raise ValueError("a model without layers")
        for i, L in enumerate(self.layers):
            own = self.layers[self.owner(i)]
            if (own.type, own.mixer, own.mlp) != (L.type, L.mixer, L.mlp):
                raise ValueError(f"layer {i} uses the weights of layer {L.weights_of}, which is another kind of layer")

    @classmethod
    def from_dict(cls, d: dict) -> "ZarinexConfig":
        mc.check_architecture(d, ARCH)
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["postln_alpha"]),
                   [LayerConfig(L["type"], L["mixer"], L.get("mlp"), L.get("weights_of")) for L in d["layers"]])

    @classmethod
    def load(cls, path: str | Path) -> "ZarinexConfig":
        return cls.from_dict(mc.read_config(path, ARCH))

    def to_dict(self) -> dict:
        return {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "postln_alpha": self.alpha,
                "layers": [L.to_dict() for L in self.layers]}

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            seen.add(i)
            i = self.layers[i].weights_of
            if not 0 <= i < len(self.layers) or i in seen:
                raise ValueError("weights_of leads to no layer with weights")
        return i


def tensor_plan(c: ZarinexConfig) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor."""
    W = c.width
    out: dict[str, tuple[int, ...]] = {"embed": (c.vocab, W), "final.norm": (W,)}
    for i, L in enumerate(c.layers):
        if L.weights_of is not None:
            continue
        p, m = f"l{i}.", L.mixer
        if L.type == "mamba1":
            I, N, R = m["inner"], m["state"], m["dt_rank"]
            mix = {"in": (2 * I, W), "conv": (I, m["conv"]), "conv.b": (I,), "x": (R + 2 * N, I), "dt": (I, R), "dt.b": (I,), "A_log": (I, N), "D": (I,), "o": (W, I)}
        elif L.type == "latent_attention":
            H, D, V, Q, K = m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            mix = {"dq": (Q, W), "dq.norm": (Q,), "uq": (H * D, Q), "dkv": (K, W), "dkv.norm": (K,), "uk": (H * D, K), "uv": (H * V, K), "g": (H * V, W),
                   "o": (W, H * V)}
        else:
            H, D, V = m["heads"], m["dim"], m["vdim"]
            mix = {"q": (H * D, W), "f": (H * D, W), "f.b": (H * D,), "lower": (H * D,), "v": (H * V, W), "norm": (V,), "o": (W, H * V)}
        out.update({p + "mix." + n: s for n, s in mix.items()})
        out.update({p + "norm1": (W,), p + "shift": (W,), p + "rg1": (W, W), p + "rg1.b": (W,)})
        if L.mlp is not None:
            out.update({p + "norm2": (W,), p + "rg2": (W, W), p + "rg2.b": (W,), p + "mlp.router": (L.experts, W), p + "mlp.router.b": (L.experts,)})
            for name, ff in [(f"e{e}", L.ff) for e in range(L.experts)] + ([("shared", L.shared_ff)] if L.shared_ff else []):
                q = p + f"mlp.{name}."
                out[q + "gate"], out[q + "up"], out[q + "down"] = (ff, W), (ff, W), (W, ff)
    return out


def random_tensors(c: ZarinexConfig, seed: int = 0, device: str = "cpu", gain: float = 1.0) -> dict[str, torch.Tensor]:
    """Random weights of the design (bf16). `gain` scales the queries and keys of the attention layers."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_plan(c).items():
        base = name.split(".", 1)[-1]
        z = torch.randn(shape, generator=g, device=device)
        if base == "mix.A_log":
            t = 0.5 + 0.8 * z
        elif base == "mix.dt.b":
            t = z - 2.5
        elif base == "mix.f.b":
            t = 2.0 + 1.5 * z
        elif base in ("mix.lower", "shift"):
            t = torch.sigmoid(z) * 0.9
        elif base in ("mix.conv.b", "mlp.router.b", "rg1.b", "rg2.b"):
            t = 0.3 * z
        elif base in ("mix.dq.norm", "mix.dkv.norm"):
            t = 1.0 + 0.1 * z
        elif len(shape) == 1:
            t = 1.0 + 0.1 * z
        elif name == "embed":
            t = z
        elif base == "mix.conv":
            t = z * shape[1] ** -0.5
        else:
            t = z * shape[1] ** -0.5 * (gain if base in ("mix.uq", "mix.uk") else 1.5 if ".mlp." in name else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


_MIXERS = {"mamba1": ml.SelectiveScanMixer, "latent_attention": ml.LatentAttentionMixer, "hgrn2": ml.HGRN2Mixer}


def _experts(L: LayerConfig, w: dict, out_gate: torch.Tensor, dtype, device) -> ml.RoutedExperts:
    up, down, gate = ([w[f"e{e}.{n}"] for e in range(L.experts)] for n in ("up", "down", "gate"))
    shared = ml.SwiGLU({n: w["shared." + n] for n in ("gate", "up", "down")}, dtype, device, name="_shared") if L.shared_ff else None
    # the softmax over the chosen logits is the renormed softmax over all of them
    router = ml.mo.Router(L.experts, L.top, score="softmax", renorm=True, on_output=True)
    return ml.RoutedExperts(w["router"], up, down, router, dtype, device, gate=gate, bias=w["router.b"], shared=shared, out_gate=out_gate)


def build_model(c: ZarinexConfig, tensors: dict[str, torch.Tensor], *, dtype: torch.dtype = torch.bfloat16, device: str = "cuda",
                slots: int = 8, pages: int = 64) -> ml.MixerModel:
    """Weights in the kernels' layout, with room for `slots` requests and `pages` pages of their positions."""
    mc.check_dtype(dtype)
    mc.check_tensors(tensor_plan(c), tensors)
    f32 = lambda n: tensors[n].float().to(device)
    sub = lambda p: {n[len(p):]: t for n, t in tensors.items() if n.startswith(p)}
    own: dict[int, ml.MixerLayer] = {}
    for i, L in enumerate(c.layers):
        if L.weights_of is not None:
            continue
        p = f"l{i}."
        room = (pages, pages * ml.mo.PAGE) if L.type in ml.PAGED else (slots,)
        mixer = _MIXERS[L.type](sub(p + "mix."), L.mixer, c.eps, dtype, device, *room, beside=[("gate", tensors[p + "rg1"])])
        layer = ml.MixerLayer(mixer, f32(p + "norm1"), shift=f32(p + "shift"), before=torch.zeros(slots, c.width, device=device), gate_b=(f32(p + "rg1.b"), None))
        if L.mlp is not None:
            layer.mlp = _experts(L, sub(p + "mlp."), tensors[p + "rg2"], dtype, device)
            layer.norm2, layer.gate_b = f32(p + "norm2"), (layer.gate_b[0], f32(p + "rg2.b"))
        own[i] = layer
    layers = [own[i] if L.weights_of is None else own[c.owner(i)].again() for i, L in enumerate(c.layers)]
    return ml.MixerModel(c.vocab, c.width, c.eps, dtype, tensors["embed"].to(torch.bfloat16).contiguous().to(device), layers, f32("final.norm"),
                         ml.FusedLinear([("head", tensors["embed"])], dtype, device), plus_one=False,
                         post=ml.PostSum(c.alpha, ml.sinusoid_frequencies(c.width).to(device)))


def build_runtime(path, **kw):
    """Runtime over a checkpoint folder (see `mixer_checkpoint.open_runtime`)."""
    return mc.open_runtime(path, ZarinexConfig.load, build_model, **kw)
