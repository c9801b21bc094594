"""Plain, slow restatement of a decoder made of mixer layers (matrix-memory LSTM, gated linear attention, windowed latent
attention with sinks, SwiGLU, sandwich norms): one function per mechanism, token by token, written from the equations and
sharing nothing with the product code. Weights are a dict name -> tensor; everything runs in the dtype of the weights
given (the tests use float64).

`MUTATE` names a deliberate fault for tests that check that a comparison would notice it (empty set: none).
"""
from __future__ import annotations

import math

import torch

MUTATE: set[str] = set()


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    return rms(x, eps) * (1 + w)


def yarn_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """Per-pair angular frequencies (float64) and the factor on cos and sin."""
    d, base = rot["dims"], float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / d) for i in range(d // 2)], dtype=torch.float64)
    s = rot.get("scaling")
    if s is None:
        return f, 1.0

    def turn_dim(t):
        return d * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(turn_dim(s["fast"])), 0)
    hi = min(math.ceil(turn_dim(s["slow"])), d - 1)
    out = []
    for i in range(d // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(float(f[i]) / s["factor"] * r + float(f[i]) * (1 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def rotate_half(x, pos: int, rot: dict):
    """x [..., dims]: pairs (i, i + dims / 2)."""
    f, mag = yarn_frequencies(rot)
    a = pos * f
    c, s = (torch.cos(a) * mag).to(x.dtype), (torch.sin(a) * mag).to(x.dtype)
    h = rot["dims"] // 2
    u, v, rest = x[..., :h], x[..., h:2 * h], x[..., 2 * h:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], -1)


def silu(z):
    return z / (1 + torch.exp(-z))


def mlstm_step(w: dict, m: dict, eps: float, h, st: dict):
    """One token of the matrix memory. st: {} at the start of a sequence."""
    H, D, V, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (w["q"] @ h).view(H, D) * D ** -0.5
    k = (w["k"] @ h).view(H, D)
    v = (w["v"] @ h).view(H, V)
    gi = cap * torch.tanh((w["i"] @ h + w["i.b"]) / cap)
    gf = torch.nn.functional.logsigmoid(cap * torch.tanh((w["f"] @ h + w["f.b"]) / cap))
    if not st:
        st.update(S=h.new_zeros(H, D, V), n=h.new_zeros(H, D), m=h.new_zeros(H))
    mt = torch.maximum(gf + st["m"], gi)
    a, b = torch.exp(gf + st["m"] - mt), torch.exp(gi - mt)
    st["S"] = a[:, None, None] * st["S"] + b[:, None, None] * k[:, :, None] * v[:, None, :]
    st["n"] = a[:, None] * st["n"] + b[:, None] * k
    st["m"] = mt
    num = torch.einsum("hdv,hd->hv", st["S"], q)
    den = torch.maximum((st["n"] * q).sum(-1).abs(), torch.exp(-mt)) + 1e-6
    o = rms(num / den[:, None], eps).reshape(H * V) * w["norm"]
    return w["o"] @ (o * torch.sigmoid(w["g"] @ h))


def gla_step(w: dict, m: dict, eps: float, h, st: dict):
    H, D, V, tau = m["heads"], m["dim"], m["vdim"], m["tau"]
    q = (w["q"] @ h).view(H, D) * D ** -0.5
    k = (w["k"] @ h).view(H, D)
    v = (w["v"] @ h).view(H, V)
    alpha = torch.sigmoid(w["a2"] @ (w["a1"] @ h) + w["a2.b"]).view(H, D) ** (1.0 / tau)
    if not st:
        st.update(S=h.new_zeros(H, D, V))
    st["S"] = alpha[:, :, None] * st["S"] + k[:, :, None] * v[:, None, :]
    o = torch.einsum("hdv,hd->hv", st["S"], q)
    o = (rms(o, eps) * w["norm"]).reshape(H * V)
    return w["o"] @ (o * silu(w["g"] @ h))


def latent_attention_step(w: dict, m: dict, eps: float, h, st: dict, pos: int):
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (w["q"] @ h).view(H, D + R)
    d = w["dkv"] @ h
    c = rms(d[:K], eps) * w["dkv.norm"]
    kr = rotate_half(d[K:], pos, m["rot"])
    st.setdefault("c", []).append(c)
    st.setdefault("kr", []).append(kr)
    window = (m.get("mask") or {}).get("size")
    if window is not None and "window" in MUTATE:
        window += 1
    first = 0 if window is None else max(0, pos - window + 1)
    C, KR = torch.stack(st["c"][first:]), torch.stack(st["kr"][first:])
    kn = (C @ w["uk"].t()).view(-1, H, D)
    vv = (C @ w["uv"].t()).view(-1, H, V)
    qr = rotate_half(q[:, D:], pos, m["rot"])
    s = (torch.einsum("hd,thd->ht", q[:, :D], kn) + torch.einsum("hr,tr->ht", qr, KR)) * m["scale"]
    sink = w["sink"] if "sink" not in MUTATE else torch.full_like(w["sink"], -1e30)
    mx = torch.maximum(s.max(-1).values, sink)
    e = torch.exp(s - mx[:, None])
    p = e / (e.sum(-1) + torch.exp(sink - mx))[:, None]
    return w["o"] @ torch.einsum("ht,thv->hv", p, vv).reshape(H * V)


MIXERS = {"mlstm": lambda w, m, eps, h, st, pos: mlstm_step(w, m, eps, h, st),
          "gla": lambda w, m, eps, h, st, pos: gla_step(w, m, eps, h, st),
          "latent_attention": latent_attention_step}


def swiglu(w: dict, h):
    return w["down"] @ (silu(w["gate"] @ h) * (w["up"] @ h))


class PlainModel:
    """Token by token; `config` is the parsed config.json, `tensors` the checkpoint."""

    def __init__(self, config: dict, tensors: dict, dtype=torch.float64):
        self.c = config
        self.t = {k: v.to(dtype) for k, v in tensors.items()}

    def sub(self, prefix: str) -> dict:
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def new_state(self) -> dict:
        return {"pos": 0, "layers": [{} for _ in self.c["layers"]]}

    def step(self, state: dict, token: int, layers_out: list | None = None):
        eps = self.c["norm"]["eps"]
        x = self.t["embed"][token].clone()
        for i, L in enumerate(self.c["layers"]):
            p = f"l{i}."
            y = MIXERS[L["type"]](self.sub(p + "mix."), L["mixer"], eps, norm_around_zero(x, self.t[p + "norm1"], eps),
                                  state["layers"][i], state["pos"])
            x = x + norm_around_zero(y, self.t[p + "norm1b"], eps)
            if L.get("mlp") is not None:
                y = swiglu(self.sub(p + "mlp."), norm_around_zero(x, self.t[p + "norm2"], eps))
                x = x + norm_around_zero(y, self.t[p + "norm2b"], eps)
            if layers_out is not None:
                layers_out.append(x.clone())
        state["pos"] += 1
        return self.t["head"] @ norm_around_zero(x, self.t["final.norm"], eps)

    def logits(self, tokens) -> torch.Tensor:
        st = self.new_state()
        return torch.stack([self.step(st, int(t)) for t in tokens])

    def generate(self, prompt, n: int) -> list[int]:
        st = self.new_state()
        z = None
        for t in prompt:
            z = self.step(st, int(t))
        out = []
        for _ in range(n):
            out.append(int(torch.argmax(z)))
            z = self.step(st, out[-1])
        return out
