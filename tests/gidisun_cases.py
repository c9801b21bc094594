"""Small random models of the Gidisun design for the tests (sizes chosen so that nothing is equal by accident), and the fake
runtime that lets the scheduler and the servers run on the oracle without a GPU."""
from __future__ import annotations

import mixer_reference as mr
import torch

from pocketllm_b200.models import gidisun as gd
from pocketllm_b200.runtime.mixer_runtime import StepEntry  # noqa: F401
from pocketllm_b200.runtime.request_cache import RequestCache


def mlstm(heads=3, dim=20, vdim=28, cap=7.0, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": ff and {"kind": "dense", "ff": ff}}


def gla(heads=5, dim=24, vdim=18, tau=9.0, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": ff and {"kind": "dense", "ff": ff}}


def latent(heads=3, dim=22, rot=12, vdim=26, rank=40, window=29, scale=0.19, base=5000.0, scaling=True, ff=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = {"factor": 3.0, "original": 300, "fast": 20.0, "slow": 1.5}
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": r}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": ff and {"kind": "dense", "ff": ff}}


def config(layers, vocab=83, width=72, eps=3e-5) -> dict:
    return {"architecture": gd.ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def tensors(cfg: dict, seed=0, rank=5, gain=1.5) -> dict:
    return gd.random_tensors(gd.GidisunConfig.from_dict(cfg), seed, decay_rank=rank, gain=gain)


def tokens(n: int, vocab: int, seed: int, low: int = 0) -> list[int]:
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(low, vocab, (n,), generator=g).tolist()


BEACON = 0     # token whose key stands out


def beacon_tensors(cfg: dict, seed=0) -> dict:
    """Weights under which every other token's query meets the key of token BEACON with a score far above all others, in the
    first layer (latent attention): what one key out of hundreds adds is then visible in the logits."""
    t = tensors(cfg, seed, gain=0.3)
    m = cfg["layers"][0]["mixer"]
    H, D, R, K = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    e = t["embed"].float()
    e[:, 0] = 0.0
    e[:, 1] = 3.0
    e[BEACON] = 0.0
    e[BEACON, 0] = 5.0
    q = t["l0.mix.q"].float().view(H, D + R, -1)
    q[:, 0] = 0.0
    q[:, 0, 1] = 1.0
    dkv, uk = t["l0.mix.dkv"].float(), t["l0.mix.uk"].float().view(H, D, K)
    dkv[0] = 0.0
    dkv[0, 0] = 2.0
    uk[:, 0] = 0.0
    uk[:, 0, 0] = 12.0 / (3.0 * m["scale"] * K ** 0.5)
    new = {"embed": e, "l0.mix.q": q.reshape(H * (D + R), -1), "l0.mix.dkv": dkv, "l0.mix.uk": uk.reshape(H * D, K),
           "l0.mix.sink": torch.linspace(-1.0, 5.0, H)}
    t.update({k: v.to(torch.bfloat16) for k, v in new.items()})
    return t


class OracleRuntime:
    """An oracle behind the interface of `MixerRuntime` (CPU, float64)."""

    def __init__(self, cfg: dict, weights: dict, max_requests=3, pages=12, page=16, plain=mr.PlainModel):
        self.m, self.vocab, self.max_requests, self.max_tokens = plain(cfg, weights), cfg["vocab"], max_requests, pages * page
        self.cache = RequestCache(max_requests, pages, page, device=None)
        self.st: dict = {}
        self.calls: list[list[int]] = []
        self.fail_next = False

    def check_status(self):
        pass

    def release(self, rid):
        self.cache.release(rid)
        self.st.pop(rid, None)

    def step(self, entries):
        if self.fail_next:
            self.fail_next = False
            raise RuntimeError("scripted step failure")
        self.calls.append([len(e.tokens) for e in entries])
        self.cache.reserve({e.rid: self.cache.length.get(e.rid, 0) + len(e.tokens) for e in entries})
        out = []
        for e in entries:
            st = self.st.setdefault(e.rid, self.m.new_state())
            z = [self.m.step(st, t) for t in e.tokens]
            out += [z[w] for w in e.want]
            self.cache.advance(e.rid, len(e.tokens))
        return torch.stack(out).float() if out else torch.empty(0, self.vocab)

    def decode_greedy(self, rids, toks, steps):
        outs = [[] for _ in rids]
        for _ in range(steps):
            z = self.step([StepEntry(r, [t], (0,)) for r, t in zip(rids, toks)])
            toks = z.argmax(-1).tolist()
            for o, t in zip(outs, toks):
                o.append(t)
        return outs
