"""Small random models of the Zemozen design for the tests (sizes chosen so that nothing is equal by accident)."""
from __future__ import annotations

import torch
from gidisun_cases import BEACON, tokens  # noqa: F401

from pocketllm_b200.models import zemozen as zm


def moe(experts=5, identity=2, top=3, ff=36):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def heads(heads=6, kv=2, dim=22, vdim=26, rot=10, base=700.0, factor=None, window=29, scale=0.21):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if factor:
            m["rot"]["scaling"] = {"factor": factor}
    if window:
        m["mask"] = {"size": window}
    return m


def attention(mlp=None, v_mix=True, factor=3.0, **kw):
    m = heads(factor=factor, **kw)
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m, "mlp": mlp}


def parallel(mlp=None, cap=2.5, scales=(0.7, 1.3), left=None, heads_=6, vdim=10, state=18, groups=3, conv=4, parts=4):
    m = {"left": heads(**{"heads": 4, "kv": 2, "dim": 18, "vdim": 14, "rot": 8, "window": 37, "scale": 0.4, **(left or {})}) | {"softcap": cap},
         "right": {"heads": heads_, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": parts},
         "left_scale": scales[0], "right_scale": scales[1]}
    return {"type": "parallel", "mixer": m, "mlp": mlp}


def config(layers, vocab=83, width=72, eps=3e-5, scale=2.5, mult=0.6) -> dict:
    return {"architecture": zm.ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "residual_mult": mult,
            "layers": layers}


FULL = config([parallel(moe()), attention(moe(experts=4, identity=1, top=2)), attention(v_mix=False, window=64, kv=3, vdim=40),
               parallel(moe(experts=3, identity=0, top=2, ff=150), left={"window": 65, "kv": 1, "dim": 40, "vdim": 130, "rot": 40, "factor": 2.0},
                        heads_=4, vdim=33, state=70, groups=1, conv=3, parts=1, scales=(1.0, 0.4)),
               attention(moe(experts=2, identity=3, top=1), factor=None)], vocab=101, width=88, mult=0.45)


def tensors(cfg: dict, seed=0, gain=1.5) -> dict:
    return zm.random_tensors(zm.ZemozenConfig.from_dict(cfg), seed, gain=gain)


def clear_routes(cfg: dict, t: dict, levels=(8.0, 5.0, 2.5, 1.1)) -> dict:
    """Weights under which no routing decision is close, so that 16-bit rounding cannot turn one: the first channels of the
    residual stream hold a pattern of the token that no mixer and no expert writes to (an identity only makes it larger), and the
    routers read mostly that. The corrections turn some decisions."""
    t = dict(t)
    n = max([L["mlp"]["router"]["experts"] + L["mlp"]["router"].get("identity", 0) for L in cfg["layers"] if L["mlp"]], default=0)
    e = t["embed"].float()
    e[:, :n] = 0.0
    for v in range(cfg["vocab"]):
        for j, level in enumerate(levels[:n]):
            e[v, (v + j * (1 + v // n % max(1, n // 3))) % n] = level / cfg["embedding"]["scale"]
    t["embed"] = e.to(torch.bfloat16)
    for name in list(t):
        if name.endswith((".o", ".down")):
            w = t[name].clone()
            w[:n] = 0
            t[name] = w
        elif name.endswith(".router"):
            w = t[name].float() * 0.02
            w[:, :n] = 0.0
            for c in range(n):
                w[c % w.shape[0], c] = 0.4
            t[name] = w.to(torch.bfloat16)
        elif name.endswith(".correction"):
            w = torch.zeros_like(t[name])
            w[0] = 0.5
            t[name] = w
        elif name.endswith((".norm1", ".norm2")):
            w = t[name].clone()
            w[:n] = 1.0
            t[name] = w
    return t


def beacon_tensors(cfg: dict, seed=0) -> dict:
    """Weights under which every other token's query meets the key of token BEACON with a score far above all others, in every head
    of the first layer's attention (with an unrotated last dimension): what one key out of hundreds adds is then visible in the
    logits."""
    t = tensors(cfg, seed, gain=0.3)
    L, W, esc = cfg["layers"][0], cfg["width"], cfg["embedding"]["scale"]
    m, p = (L["mixer"], "l0.mix.") if L["type"] == "attention" else (L["mixer"]["left"], "l0.mix.left.")
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    assert m.get("rot", {"dims": 0})["dims"] < D
    e = t["embed"].float()
    e[:, 0] = 0.0
    e[:, 1] = 3.0 / esc
    e[BEACON] = 0.0
    e[BEACON, 0] = 5.0 / esc
    q, k, qn, kn = t[p + "q"].float().view(H, D, W), t[p + "k"].float().view(G, D, W), t[p + "q.norm"].float(), t[p + "k.norm"].float()
    q[:, -1] = 0.0
    q[:, -1, 1] = 3.0
    k[:, -1] = 0.0
    k[:, -1, 0] = 3.0
    qn[-1] = 1.0
    kn[-1] = 14.0 / (D * m["scale"])
    new = {"embed": e, p + "q": q.reshape(-1, W), p + "k": k.reshape(-1, W), p + "q.norm": qn, p + "k.norm": kn}
    t.update({n: v.to(torch.bfloat16) for n, v in new.items()})
    return t
