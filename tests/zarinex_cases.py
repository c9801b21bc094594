"""Small random models of the Zarinex design for the tests (sizes chosen so that nothing is equal by accident)."""
from __future__ import annotations

import torch
from gidisun_cases import BEACON, tokens  # noqa: F401

from pocketllm_b200.models import zarinex as zx


def moe(experts=5, top=2, ff=36, shared=52):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared} if shared else None}


def scan(mlp=None, inner=60, state=10, rank=7, conv=4):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}, "mlp": mlp}


def latent(mlp=None, heads=3, dim=22, vdim=26, q_rank=30, kv_rank=41, scale=0.23):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}, "mlp": mlp}


def forget(mlp=None, heads=5, dim=20, vdim=28):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def again(layer: dict, of: int) -> dict:
    return layer | {"weights_of": of}


def config(layers, vocab=83, width=72, eps=3e-5, alpha=1.7) -> dict:
    return {"architecture": zx.ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


_A, _B, _C = scan(moe()), latent(moe(experts=4, top=3, ff=20, shared=130)), forget(moe(experts=3, top=1, ff=150, shared=None))
FULL = config([_A, _B, again(_A, 0), _C, forget(heads=2, dim=37, vdim=9), again(_C, 3), again(_B, 1), scan(moe(experts=2, top=2), inner=33, state=21, rank=40, conv=3),
               again(_A, 2)], vocab=101, width=88, alpha=2.3)


def tensors(cfg: dict, seed=0, gain=1.5) -> dict:
    return zx.random_tensors(zx.ZarinexConfig.from_dict(cfg), seed, gain=gain)


def clear_routes(cfg: dict, t: dict, levels=(14.0, 10.5, 7.0, 3.5)) -> dict:
    """Weights under which no routing decision is close, so that 16-bit rounding cannot turn one: the first channels of the residual
    stream hold a pattern of the token, far above the sinusoids, that no mixer and no expert writes to; the routers read mostly that, and
    their biases turn some decisions. The output matrix, which is the embedding table, sees little of the pattern."""
    t = dict(t)
    n = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if L["mlp"]], default=0)
    e = t["embed"].float()
    e[:, :n] = 0.0
    for v in range(cfg["vocab"]):
        for j, level in enumerate(levels[:n]):
            e[v, (v + j) % n] = level
    t["embed"] = e.to(torch.bfloat16)
    for name in list(t):
        w = t[name].clone()
        if name.endswith((".o", ".down")):
            w = w.float() * 1.5
            w[:n] = 0
        elif name.endswith(".router"):
            w = w.float() * 0.005
            w[:, :n] = 0.0
            for c in range(w.shape[0]):
                w[c, c] = 0.6
        elif name.endswith(".router.b"):
            w = torch.zeros_like(w)
            w[0] = 6.0
        elif name.endswith((".norm1", ".norm2")):
            w[:n] = 1.6      # the pattern is not to fade
        elif name == "final.norm":
            w[:n] = 0.05
        t[name] = w.to(torch.bfloat16)
    return t


def beacon_tensors(cfg: dict, seed=0) -> dict:
    """Weights under which every other token's query meets the key of token BEACON with a score far above all others, in every head of
    the first layer (latent attention): what one key out of hundreds adds is then visible in the logits. The marks lie in the last two
    channels, where the sinusoids hardly move, and pass the token shift unmixed."""
    t = tensors(cfg, seed, gain=0.3)
    m, W = cfg["layers"][0]["mixer"], cfg["width"]
    assert cfg["layers"][0]["type"] == "latent_attention" and W % 2 == 0
    H, D = m["heads"], m["dim"]
    e = t["embed"].float()
    e[:, W - 2] = 0.0
    e[:, W - 1] = 3.0
    e[BEACON] = 0.0
    e[BEACON, W - 2] = 8.0
    dq, dkv, uq, uk, sh = (t["l0." + n].float() for n in ("mix.dq", "mix.dkv", "mix.uq", "mix.uk", "shift"))
    sh[W - 2:] = 0.0
    dq[:, W - 2:] = 0.0
    dq[0], dkv[:, W - 2:], dkv[0] = 0.0, 0.0, 0.0
    dq[0, W - 1] = dkv[0, W - 2] = 3.0
    uq, uk = uq.view(H, D, -1), uk.view(H, D, -1)
    uq[:, 0] = uk[:, 0] = 0.0
    uq[:, 0, 0] = 1.0
    uk[:, 0, 0] = 0.5 / m["scale"]
    o, gb = t["l0.mix.o"].float() * 4.0, t["l0.rg1.b"].float() + 2.0
    new = {"l0.mix.o": o, "l0.rg1.b": gb, "embed": e, "l0.mix.dq": dq, "l0.mix.dkv": dkv, "l0.mix.uq": uq.reshape(H * D, -1), "l0.mix.uk": uk.reshape(H * D, -1), "l0.shift": sh}
    t.update({n: v.to(torch.bfloat16) for n, v in new.items()})
    return t
