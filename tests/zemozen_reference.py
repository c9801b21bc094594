"""Plain, slow restatement of the Zemozen design (windowed attention with head norms, mixed values and head gates; attention with
capped scores and a sink beside a state-space recurrence; routed experts of which some return their input): one function per
mechanism, token by token, written from the equations and sharing nothing with the product code. Weights are a dict name ->
tensor; everything runs in the dtype of the weights given (the tests use float64).

`MUTATE` names a deliberate fault for tests that check that a comparison would notice it (empty set: none).
"""
from __future__ import annotations

import torch
from mixer_reference import rms, silu

MUTATE: set[str] = set()


def turn(x, pos: int, rot: dict | None, neighbours: bool):
    """x [heads, dim]: the first rot.dims of every head turn, the rest pass. A pair is (i, i + dims / 2), or (2i, 2i + 1)."""
    if not rot or rot["dims"] == 0:
        return x
    n = rot["dims"]
    i = torch.arange(n // 2, dtype=torch.float64)
    f = float(rot["base"]) ** (-2.0 * i / n)
    if rot.get("scaling"):
        f = f / float(rot["scaling"]["factor"])
    c, s = torch.cos(pos * f).to(x.dtype), torch.sin(pos * f).to(x.dtype)
    a, b = (slice(0, n, 2), slice(1, n, 2)) if neighbours else (slice(0, n // 2), slice(n // 2, n))
    out = x.clone()
    out[..., a], out[..., b] = x[..., a] * c - x[..., b] * s, x[..., b] * c + x[..., a] * s
    return out


def visible_from(pos: int, mask: dict | None) -> int:
    if not mask:
        return 0
    return max(0, pos - mask["size"] + 1 - ("window" in MUTATE))


def head_norm(x, w, eps):
    return x if "head_norm" in MUTATE else rms(x, eps) * w


def cached_attention(w: dict, m: dict, eps: float, h, st: dict, pos: int, v, neighbours: bool):
    """Appends this token and yields (head, scores over the visible positions, their values)."""
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = turn(head_norm((w["q"] @ h).view(H, D), w["q.norm"], eps), pos, m.get("rot"), neighbours)
    k = turn(head_norm((w["k"] @ h).view(G, D), w["k.norm"], eps), pos, m.get("rot"), neighbours)
    st.setdefault("k", []).append(k)
    st.setdefault("v", []).append(v)
    first = visible_from(pos, m.get("mask"))
    K, V = torch.stack(st["k"][first:]), torch.stack(st["v"][first:])
    for i in range(H):
        g = i // (H // G)
        yield i, (K[:, g] @ q[i]) * m["scale"], V[:, g]


def attention_step(w: dict, m: dict, eps: float, h, st: dict, pos: int, shared: dict):
    """`shared` holds what this token's earlier layers leave for later ones: the first mixing layer's values."""
    v = (w["v"] @ h).view(m["kv_heads"], m["vdim"])
    if m.get("v_mix"):
        if "v" not in shared:
            shared["v"] = v
        elif "v_mix" not in MUTATE:
            v = (1 - w["vmix"]) * v + w["vmix"] * shared["v"]
    gate = torch.sigmoid(w["g"] @ h)
    outs = []
    for i, s, V in cached_attention(w, m, eps, h, st, pos, v, neighbours=False):
        o = torch.softmax(s, 0) @ V
        outs.append(o if "gate" in MUTATE else o * gate[i])
    return w["o"] @ torch.cat(outs)


def capped_sink_attention_step(w: dict, m: dict, eps: float, h, st: dict, pos: int):
    v = (w["v"] @ h).view(m["kv_heads"], m["vdim"])
    outs = []
    for _, s, V in cached_attention(w, m, eps, h, st, pos, v, neighbours="pairs" not in MUTATE):
        if "cap" not in MUTATE:
            s = m["softcap"] * torch.tanh(s / m["softcap"])
        top = torch.clamp(s.max(), min=0)
        e = torch.exp(s - top)
        den = e.sum() + (0 if "sink" in MUTATE else torch.exp(-top))
        outs.append((e / den) @ V)
    return w["o"] @ torch.cat(outs)


def state_space_step(w: dict, m: dict, eps: float, h, st: dict):
    """One token of Mamba-2: short causal convolution, scalar decay per head, state [heads, N, vdim]."""
    H, V, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    inner = H * V
    p = w["in"] @ h
    z, xbc, dt = p[:inner], p[inner:inner + inner + 2 * G * N], p[-H:]
    past = st.setdefault("past", [torch.zeros_like(xbc)] * (taps - 1))
    line = past + [xbc]
    y = w["conv.b"].clone()
    for j in range(taps):
        y = y + w["conv"][:, j] * line[j]
    st["past"] = line[1:]
    y = silu(y)
    x, B, C = y[:inner].view(H, V), y[inner:inner + G * N].view(G, N), y[inner + G * N:].view(G, N)
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
    if "S" not in st:
        st["S"] = h.new_zeros(H, N, V)
    a = torch.exp(-torch.exp(w["A_log"]) * dt)
    outs = []
    for i in range(H):
        g = i // (H // G) if "groups" not in MUTATE else 0
        st["S"][i] = a[i] * st["S"][i] + dt[i] * B[g][:, None] * x[i][None, :]
        outs.append(st["S"][i].t() @ C[g] + (0 if "skip" in MUTATE else w["D"][i] * x[i]))
    y = torch.cat(outs) * silu(z)
    y = rms(y.view(m["norm_groups"], -1), eps).reshape(-1) * w["norm"]
    return w["o"] @ y


def part(w: dict, side: str) -> dict:
    return {k[len(side) + 1:]: t for k, t in w.items() if k.startswith(side + ".")}


def parallel_step(w: dict, m: dict, eps: float, h, st: dict, pos: int):
    a = capped_sink_attention_step(part(w, "left"), m["left"], eps, h, st.setdefault("left", {}), pos)
    b = state_space_step(part(w, "right"), m["right"], eps, h, st.setdefault("right", {}))
    return m["left_scale"] * a + m["right_scale"] * b


def route(w: dict, m: dict, h) -> list[tuple[int, torch.Tensor]]:
    """(expert, weight) of the chosen experts: largest corrected softmax scores, weighted by the uncorrected ones, normed."""
    s = torch.softmax(w["router"] @ h, 0)
    c = s if "correction" in MUTATE else s + w["correction"]
    top = sorted(range(len(s)), key=lambda e: (-float(c[e]), e))[:m["router"]["top"]]
    total = sum(s[e] for e in top) + 1e-20
    return [(e, s[e] / total) for e in top]


def experts(w: dict, m: dict, h):
    y = torch.zeros_like(h)
    for e, s in route(w, m, h):
        if e >= m["router"]["experts"]:
            y = y + (0 if "identity" in MUTATE else s * h)
        else:
            y = y + s * (w[f"e{e}.down"] @ (silu(w[f"e{e}.gate"] @ h) * (w[f"e{e}.up"] @ h)))
    return y


class PlainModel:
    """Token by token; `config` is the parsed config.json, `tensors` the checkpoint."""

    def __init__(self, config: dict, tensors: dict, dtype=torch.float64):
        self.c = config
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.w = [(self._sub(f"l{i}.mix."), self._sub(f"l{i}.mlp.")) for i in range(len(config["layers"]))]

    def _sub(self, prefix: str) -> dict:
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def new_state(self) -> dict:
        return {"pos": 0, "layers": [{} for _ in self.c["layers"]]}

    def norm(self, x, name: str):
        return rms(x, self.c["norm"]["eps"]) * self.t[name]

    def step(self, state: dict, token: int, layers_out: list | None = None):
        eps, mult, pos = self.c["norm"]["eps"], self.c["residual_mult"], state["pos"]
        if "residual" in MUTATE:
            mult = 1.0
        x, shared = self.t["embed"][token] * self.c["embedding"]["scale"], {}
        for i, (L, (wm, wf), st) in enumerate(zip(self.c["layers"], self.w, state["layers"])):
            h = self.norm(x, f"l{i}.norm1")
            if L["type"] == "attention":
                y = attention_step(wm, L["mixer"], eps, h, st, pos, shared)
            else:
                y = parallel_step(wm, L["mixer"], eps, h, st, pos)
            x = x + mult * y
            if L.get("mlp") is not None:
                x = x + mult * experts(wf, L["mlp"], self.norm(x, f"l{i}.norm2"))
            if layers_out is not None:
                layers_out.append(x.clone())
        state["pos"] += 1
        return self.t["head"] @ self.norm(x, "final.norm")

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
