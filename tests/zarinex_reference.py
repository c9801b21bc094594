"""Plain, slow restatement of the Zarinex design (norm after the sum, token shift, gated sublayers; selective scan, latent
attention without positions, linear attention whose forget gate decides what is written; routed experts beside a shared one): one
function per mechanism, token by token, written from the equations and sharing nothing with the product code. Weights are a dict
name -> tensor; everything runs in the dtype of the weights given (the tests use float64).

`MUTATE` names a deliberate fault for tests that check that a comparison would notice it (empty set: none).
"""
from __future__ import annotations

import torch
from mixer_reference import rms, silu

MUTATE: set[str] = set()


def sinusoid(pos: int, width: int, dtype):
    """Column 2i: sin(pos r^i), column 2i + 1: cos(pos r^i), with r^i = 10000^(-2i / width)."""
    out = torch.zeros(width, dtype=torch.float64)
    for c in range(width):
        a = torch.tensor(pos * 10000.0 ** (-(c - c % 2) / width), dtype=torch.float64)
        out[c] = torch.cos(a) if c % 2 else torch.sin(a)
    return out.to(dtype)


def selective_scan_step(w: dict, m: dict, eps: float, h, st: dict):
    """One token of Mamba: state [inner, state], a step size per channel."""
    inner, N, taps, rank = m["inner"], m["state"], m["conv"], m["dt_rank"]
    p = w["in"] @ h
    x, z = p[:inner], p[inner:]
    past = st.setdefault("past", [torch.zeros_like(x)] * (taps - 1))
    line = past + [x]
    y = w["conv.b"].clone()
    for j in range(taps):
        y = y + w["conv"][:, j] * line[j]
    st["past"] = line[1:]
    x = silu(y)
    d = w["x"] @ x
    dt, B, C = d[:rank], d[rank:rank + N], d[rank + N:]
    dt = torch.nn.functional.softplus(w["dt"] @ dt + w["dt.b"], threshold=1e9)
    if "S" not in st:
        st["S"] = h.new_zeros(inner, N)
    a = torch.exp(-dt[:, None] * torch.exp(w["A_log"]))
    st["S"] = a * st["S"] + (dt * x)[:, None] * B[None, :]
    y = st["S"] @ C + (0 if "skip" in MUTATE else w["D"] * x)
    return w["o"] @ (y * silu(z))


def latent_attention_step(w: dict, m: dict, eps: float, h, st: dict):
    """Queries, keys and values from latents, every earlier token visible, a sigmoid gate on the heads' outputs."""
    H, D, V = m["heads"], m["dim"], m["vdim"]
    cq = w["dq"] @ h
    if "q_norm" not in MUTATE:
        cq = rms(cq, eps) * w["dq.norm"]
    q = (w["uq"] @ cq).view(H, D)
    c = rms(w["dkv"] @ h, eps) * w["dkv.norm"]
    st.setdefault("c", []).append(c)
    C = torch.stack(st["c"])
    k, v = (C @ w["uk"].t()).view(-1, H, D), (C @ w["uv"].t()).view(-1, H, V)
    p = torch.softmax(torch.einsum("hd,thd->ht", q, k) * m["scale"], -1)
    o = torch.einsum("ht,thv->hv", p, v).reshape(H * V)
    if "out_gate" not in MUTATE:
        o = o * torch.sigmoid(w["g"] @ h)
    return w["o"] @ o


def forget_write_step(w: dict, m: dict, eps: float, h, st: dict):
    """HGRN2: what the forget gate drops from a key channel is what the value is written with."""
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q, v = silu(w["q"] @ h).view(H, D), (w["v"] @ h).view(H, V)
    low = torch.zeros_like(w["lower"]) if "lower" in MUTATE else w["lower"]
    f = (low + (1 - low) * torch.sigmoid(w["f"] @ h + w["f.b"])).view(H, D)
    if "S" not in st:
        st["S"] = h.new_zeros(H, D, V)
    st["S"] = f[:, :, None] * st["S"] + (1 - f)[:, :, None] * v[:, None, :]
    o = torch.einsum("hdv,hd->hv", st["S"], q)
    return w["o"] @ (rms(o, eps) * w["norm"]).reshape(H * V)


MIXERS = {"mamba1": selective_scan_step, "latent_attention": latent_attention_step, "hgrn2": forget_write_step}


def expert(w: dict, name: str, h):
    return w[name + ".down"] @ (silu(w[name + ".gate"] @ h) * (w[name + ".up"] @ h))


def route(w: dict, m: dict, h) -> list[tuple[int, torch.Tensor]]:
    """(expert, weight): the largest logits, weighted by the softmax over themselves."""
    z = w["router"] @ h + (0 if "router_bias" in MUTATE else w["router.b"])
    top = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[:m["router"]["top"]]
    return list(zip(top, torch.softmax(torch.stack([z[e] for e in top]), 0)))


def experts(w: dict, m: dict, h):
    y = torch.zeros_like(h)
    for e, s in route(w, m, h):
        y = y + s * expert(w, f"e{e}", h)
    if m.get("shared") and "shared" not in MUTATE:
        y = y + expert(w, "shared", h)
    return y


def token_shift(w, h, st: dict):
    """A step from this token's input towards the previous token's, element by element."""
    before = st.get("h", torch.zeros_like(h))
    st["h"] = h
    return h if "shift" in MUTATE else h + (before - h) * w


class PlainModel:
    """Token by token; `config` is the parsed config.json, `tensors` the checkpoint."""

    def __init__(self, config: dict, tensors: dict, dtype=torch.float64):
        self.c = config
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.own = []
        for i, L in enumerate(config["layers"]):
            while "weights_of" in config["layers"][i]:
                i = config["layers"][i]["weights_of"]
            self.own.append(i)
        self.w = [self._sub(f"l{i}.") for i in self.own]

    def _sub(self, prefix: str) -> dict:
        d = {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}
        part = lambda p: {k[len(p):]: v for k, v in d.items() if k.startswith(p)}
        return {"": d, "mix": part("mix."), "mlp": part("mlp.")}

    def new_state(self) -> dict:
        return {"pos": 0, "layers": [{} for _ in self.c["layers"]]}

    def add(self, x, y, w: dict, n: int):
        """norm(alpha x + sigmoid(gate of x) y)"""
        if "gated" not in MUTATE:
            y = y * torch.sigmoid(w[f"rg{n}"] @ x + w[f"rg{n}.b"])
        return rms(self.c["postln_alpha"] * x + y, self.c["norm"]["eps"]) * w[f"norm{n}"]

    def step(self, state: dict, token: int, layers_out: list | None = None):
        eps, pos = self.c["norm"]["eps"], state["pos"]
        x = self.t["embed"][token]
        if "position" not in MUTATE:
            x = x + sinusoid(pos, len(x), x.dtype)
        states = state["layers"]
        for i, (L, w) in enumerate(zip(self.c["layers"], self.w)):
            st = states[self.own[i] if "shared_state" in MUTATE else i]
            y = MIXERS[L["type"]](w["mix"], L["mixer"], eps, token_shift(w[""]["shift"], x, st), st)
            x = self.add(x, y, w[""], 1)
            if L.get("mlp") is not None:
                x = self.add(x, experts(w["mlp"], L["mlp"], x), w[""], 2)
            if layers_out is not None:
                layers_out.append(x.clone())
        state["pos"] += 1
        return self.t["embed"] @ (rms(x, eps) * self.t["final.norm"])

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
