"""What the GPU tests of mixer decoders share: feeding a runtime in portions, comparing with the oracle, traffic of unequal
requests through few slots and pages."""
from __future__ import annotations

import torch

F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 1e-4, BF16: 0.08}


def make_runtime(module, config_class, cfg, t, dtype=F32, max_requests=4, pages=24, **kw):
    from pocketllm_b200.runtime.mixer_runtime import MixerRuntime
    model = module.build_model(config_class.from_dict(cfg), t, dtype=dtype, slots=max_requests, pages=pages)
    return MixerRuntime(model, max_requests=max_requests, pages=pages, **kw)


def feed(rt, rid, toks, cuts, end=True):
    """Logits of all places of `toks`, run in portions of the given sizes (the last size repeats)."""
    from pocketllm_b200.runtime.mixer_runtime import StepEntry
    out, a, i = [], 0, 0
    while a < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - a)
        out.append(rt.step([StepEntry(rid, toks[a:a + n], range(n))]).clone())
        a, i = a + n, i + 1
    rt.check_status()
    if end:
        rt.release(rid)
    return torch.cat(out).double().cpu()


def off(got, want):
    """Per place: rms difference over the vocabulary relative to the logits' spread."""
    return ((got - want).pow(2).mean(-1).sqrt() / want.std()).max().item()


def check(got, want, dtype=F32, factor=1.0):
    e = off(got, want)
    assert e < TOL[dtype] * factor, e


def traffic(rt, seqs, live_max: int, pages: int, seed: int = 5, sizes=(1, 1, 2, 5, 8, 9, 40, 64, 90)) -> list[torch.Tensor]:
    """All requests through `live_max` slots and `pages` pages: portions beside single tokens, requests that rest for some
    steps, pages and slots used again. Logits of every place of every request."""
    from pocketllm_b200.runtime.mixer_runtime import StepEntry
    g = torch.Generator().manual_seed(seed)
    n_req, lens = len(seqs), [len(s) for s in seqs]
    at, got, live, nxt = {}, {i: [] for i in range(n_req)}, [], 0
    while nxt < n_req or live:
        while nxt < n_req and len(live) < live_max and sum(-(-lens[i] // 64) for i in live + [nxt]) <= pages:
            live.append(nxt)
            at[nxt] = 0
            nxt += 1
        entries = []
        for i in live:
            if len(live) > 1 and torch.rand(1, generator=g) < 0.2 and entries:
                continue
            n = sizes[int(torch.randint(0, len(sizes), (1,), generator=g))]
            n = min(n, lens[i] - at[i])
            entries.append(StepEntry(i, seqs[i][at[i]:at[i] + n], range(n)))
        z = rt.step(entries).double().cpu()
        a = 0
        for e in entries:
            n = len(e.tokens)
            got[e.rid].append(z[a:a + n])
            a += n
            at[e.rid] += n
            if at[e.rid] == lens[e.rid]:
                rt.release(e.rid)
                live.remove(e.rid)
    rt.check_status()
    assert rt.cache.free_pages == pages and rt.cache.free_slots == live_max
    return [torch.cat(got[i]) for i in range(n_req)]


def margin_prefix(m, prompt, n, eps):
    """Greedy continuation of the oracle up to the first near-tie."""
    st = m.new_state()
    for x in prompt:
        z = m.step(st, x)
    out = []
    for _ in range(n):
        top = torch.topk(z, 2).values
        if top[0] - top[1] < eps:
            break
        out.append(int(z.argmax()))
        z = m.step(st, out[-1])
    return out
