"""Small random models of the Pezarax design for the tests (sizes chosen so that nothing is equal by accident)."""
from __future__ import annotations

import torch
from gidisun_cases import BEACON, tokens  # noqa: F401

from pocketllm_b200.models import pezarax as pz


def moe(experts=5, top=2, ff=36):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def retention(heads=3, dim=20, vdim=28, rot=12, base=3000.0, decay=(0.6, 0.97, 0.9995), mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": [decay[i % len(decay)] for i in range(heads)]}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
    return {"type": "retention", "mixer": m, "mlp": mlp}


def attention(heads=6, kv=2, dim=22, vdim=26, rot=10, base=700.0, chunk=29, scale=0.21, diff=0.3, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
    if chunk:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(layers, vocab=83, width=72, eps=3e-5, scale=2.5, logit_scale=0.7, loop=None) -> dict:
    d = {"architecture": pz.ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "logit_scale": logit_scale,
         "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


FULL = config([retention(mlp=moe()), attention(mlp=moe()), retention(heads=2, dim=9, vdim=40, rot=4, decay=(0.9, 0.999)),
               attention(heads=3, kv=3, dim=40, vdim=130, rot=40, chunk=64, diff=0.8, scale=0.16, mlp=moe(top=1, ff=150))],
              vocab=101, width=88, loop=(1, 3, 3))


def tensors(cfg: dict, seed=0, gain=1.5) -> dict:
    return pz.random_tensors(pz.PezaraxConfig.from_dict(cfg), seed, gain=gain)


def clear_routes(cfg: dict, t: dict, levels=(7.0, 5.0, 3.2)) -> dict:
    """Weights under which no routing decision is close, so that 16-bit rounding cannot turn one: the first channels of the
    residual stream hold a pattern of the token that no layer writes to, and the routers read mostly that."""
    t = dict(t)
    n = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if L["mlp"]], default=0)
    e = t["embed"].float()
    e[:, :n] = 0.0
    for v in range(cfg["vocab"]):
        for j, level in enumerate(levels[:n]):
            e[v, (v + j * (1 + v // n % max(1, n // 3))) % n] = level / cfg["embedding"]["scale"]
    t["embed"] = e.to(torch.bfloat16)
    for name in list(t):
        if name.endswith((".mix.o", ".down")):
            w = t[name].clone()
            w[:n] = 0
            t[name] = w
        elif name.endswith(".router"):
            w = t[name].float() * 0.02
            w[:, :n] = 0.0
            for i in range(w.shape[0]):
                w[i, i] = 0.4
            t[name] = w.to(torch.bfloat16)
        elif name.endswith((".norm1", ".norm2")):
            w = t[name].clone()
            w[:n] = 1.0
            t[name] = w
    return t


def beacon_tensors(cfg: dict, seed=0, chosen_map=0) -> dict:
    """Weights under which every other token's query meets the key of token BEACON with a score far above all others, in one map
    of every head of the first layer (attention with an unrotated last dimension): what one key out of hundreds adds is then
    visible in the logits."""
    t = tensors(cfg, seed, gain=0.3)
    m, W, esc = cfg["layers"][0]["mixer"], cfg["width"], cfg["embedding"]["scale"]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    assert m.get("rot", {"dims": 0})["dims"] < D
    e = t["embed"].float()
    e[:, 0] = 0.0
    e[:, 1] = 3.0 / esc
    e[BEACON] = 0.0
    e[BEACON, 0] = 5.0 / esc
    q, k = t["l0.mix.q"].float().view(H, 2, D, W), t["l0.mix.k"].float().view(G, 2, D, W)
    q[:, chosen_map, -1] = 0.0
    q[:, chosen_map, -1, 1] = 2.0
    k[:, chosen_map, -1] = 0.0
    k[:, chosen_map, -1, 0] = 14.0 / (2.0 * 2.6 * m["scale"] * W ** 0.5)
    new = {"embed": e, "l0.mix.q": q.reshape(-1, W), "l0.mix.k": k.reshape(-1, W)}
    t.update({n: v.to(torch.bfloat16) for n, v in new.items()})
    return t
