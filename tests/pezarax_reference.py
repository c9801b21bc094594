"""Plain, slow restatement of the Pezarax design (retention, chunked differential attention, routed experts weighted at their
input, layers that run several times): one function per mechanism, token by token, written from the equations and sharing
nothing with the product code. Weights are a dict name -> tensor; everything runs in the dtype of the weights given (the
tests use float64).

`MUTATE` names a deliberate fault for tests that check that a comparison would notice it (empty set: none).
"""
from __future__ import annotations


import torch
from mixer_reference import rms, rotate_half, silu

MUTATE: set[str] = set()


def rotate_heads(x, pos: int, rot: dict | None):
    """x [heads, dim]: the first rot.dims of every head turn, the rest pass."""
    return x if rot is None or rot["dims"] == 0 else rotate_half(x, pos, rot)


def retention_step(w: dict, m: dict, eps: float, h, st: dict, pos: int):
    """One token; the state (one matrix per head) decays by a constant and takes k v^T in."""
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = rotate_heads((w["q"] @ h).view(H, D), pos, m.get("rot"))
    k = rotate_heads((w["k"] @ h).view(H, D), pos, m.get("rot")) * D ** -0.5
    v = (w["v"] @ h).view(H, V)
    if not st:
        st["S"] = h.new_zeros(H, D, V)
    a = torch.tensor(m["decay"], dtype=h.dtype)
    st["S"] = a[:, None, None] * st["S"] + k[:, :, None] * v[:, None, :]
    o = rms(torch.einsum("hdv,hd->hv", st["S"], q), eps).reshape(H * V)
    return w["o"] @ (o * silu(w["g"] @ h))


def first_visible(pos: int, mask: dict | None) -> int:
    if not mask:
        return 0
    size = mask["size"] + (1 if "chunk" in MUTATE else 0)
    return pos // size * size


def diff_lambda(w: dict, diff: float):
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def diff_attention_step(w: dict, m: dict, eps: float, h, st: dict, pos: int):
    """Two softmax maps per head over the same values; their difference is normed per head."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_heads((w["q"] @ h).view(H * 2, D), pos, m.get("rot")).view(H, 2, D)
    k = rotate_heads((w["k"] @ h).view(G * 2, D), pos, m.get("rot")).view(G, 2, D)
    st.setdefault("k", []).append(k)
    st.setdefault("v", []).append((w["v"] @ h).view(G, V))
    first = first_visible(pos, m.get("mask"))
    K, Vs = torch.stack(st["k"][first:]), torch.stack(st["v"][first:])          # [t, G, 2, D], [t, G, V]
    lam = diff_lambda(w, m["diff"])
    if "lambda" in MUTATE:
        lam = lam * 0
    outs = []
    for i in range(H):
        g = i // (H // G)
        a = []
        for c in (0, 1):
            s = (K[:, g, c] @ q[i, c]) * m["scale"]
            a.append(torch.softmax(s, 0) @ Vs[:, g])
        outs.append(rms(a[0] - lam * a[1], eps) * (1 - m["diff"]))
    return w["o"] @ torch.cat(outs)


MIXERS = {"retention": retention_step, "attention": diff_attention_step}


def route(w: dict, m: dict, h) -> list[tuple[int, torch.Tensor]]:
    """(expert, weight) of the chosen experts: the largest sigmoid scores, not renormalised."""
    s = torch.sigmoid(w["router"] @ h)
    order = sorted(range(len(s)), key=lambda e: (-float(s[e]), e))
    return [(e, s[e]) for e in order[:m["router"]["top"]]]


def experts(w: dict, m: dict, h):
    """The routing weight multiplies an expert's input."""
    y = torch.zeros_like(h)
    for e, s in route(w, m, h):
        up = torch.relu(w[f"e{e}.up"] @ (h if "weight" in MUTATE else s * h)) ** 2
        y = y + w[f"e{e}.down"] @ up * (s if "weight" in MUTATE else 1)
    return y


def layer_runs(config: dict) -> list[tuple[int, bool]]:
    """(layer, whether the embedding output is added before it) for every run of a layer, in order."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == a and "reinject" not in MUTATE) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


class PlainModel:
    """Token by token; `config` is the parsed config.json, `tensors` the checkpoint."""

    def __init__(self, config: dict, tensors: dict, dtype=torch.float64):
        self.c, self.runs = config, layer_runs(config)
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.w = [(self._sub(f"l{i}.mix."), self._sub(f"l{i}.mlp.")) for i in range(len(config["layers"]))]

    def _sub(self, prefix: str) -> dict:
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def new_state(self) -> dict:
        return {"pos": 0, "runs": [{} for _ in self.runs]}

    def norm(self, x, name: str):
        return rms(x, self.c["norm"]["eps"]) * self.t[name]

    def step(self, state: dict, token: int, layers_out: list | None = None):
        eps = self.c["norm"]["eps"]
        e = self.t["embed"][token] * self.c["embedding"]["scale"]
        x = e.clone()
        for (i, again), st in zip(self.runs, state["runs"]):
            L, (wm, wf) = self.c["layers"][i], self.w[i]
            if again:
                x = x + e
            x = x + MIXERS[L["type"]](wm, L["mixer"], eps, self.norm(x, f"l{i}.norm1"), st, state["pos"])
            if L.get("mlp") is not None:
                x = x + experts(wf, L["mlp"], self.norm(x, f"l{i}.norm2"))
            if layers_out is not None:
                layers_out.append(x.clone())
        state["pos"] += 1
        return self.t["head"] @ self.norm(x, "final.norm") * self.c["logit_scale"]

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
