"""Zarinex on the GPU against the plain oracle (float64, token by token): every mechanism alone, prompts, portions, mixed batches, reused
pages and slots, a far key among many, long memories, long decoding, unusual sizes, generation through the scheduler, the CLI."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch
import zarinex_reference as zr
from mixer_checks import BF16, F32, check, feed, make_runtime, margin_prefix, traffic
from mixer_reference import rms
from zarinex_cases import BEACON, FULL, again, beacon_tensors, clear_routes, config, forget, latent, moe, scan, tensors, tokens

from pocketllm_b200.models import zarinex as zx
from pocketllm_b200.server.engine import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def runtime(cfg, t, dtype=F32, **kw):
    return make_runtime(zx, zx.ZarinexConfig, cfg, t, dtype, **kw)


_memo: dict = {}


def oracle(cfg, t, seq, key):
    k = (key, len(seq))
    if k not in _memo:
        _memo[k] = zr.PlainModel(cfg, t).logits(seq)
    return _memo[k]


# ---- kernels ----

PORTIONS = [(3, 0, 2), (1, 5, 0), (1, 0, 4), (9, 64, 1), (2, 1, 3)]      # tokens, first position, slot


def _batch(scale: int = 1):
    dev = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda")
    pos, slot, behind = [], [], []
    for n, p, s in PORTIONS:
        n *= scale
        pos += range(p, p + n)
        slot += [s] * n
        behind += range(n - 1, -1, -1)
    return dev(pos), dev(slot), dev(behind)


@pytest.mark.parametrize("hdt", [F32, BF16])
@pytest.mark.parametrize("W,scale", [(24, 1), (301, 1), (2048, 1), (2048, 90), (301, 90), (5000, 1), (8192, 5), (16384, 1)])
def test_steps_with_the_norm_behind_the_sum(W, scale, hdt):
    """The residual step in all its forms: gate, rows of experts and a second output, token shift over portions, what is kept for the next
    step, the final norm of listed rows."""
    from pocketllm_b200.ops import mixer_ops as mo
    pos, slot, behind = _batch(scale)
    T, eps, alpha = len(pos), 1e-3, 1.9
    r = lambda *s: torch.randn(*s, device="cuda")
    x, y, y2, gate = r(T, W), r(2 * T, W + 4), r(T, W + 8), r(T, W + 12)
    b, w, wf, shift, before = r(W), r(W), r(W), torch.rand(W, device="cuda"), r(6, W)
    place = torch.randint(-1, 2 * T, (T, 2), dtype=torch.int32, device="cuda")
    picked = torch.where((place >= 0)[..., None], y[place.clamp(min=0).long(), :W], torch.zeros((), device="cuda")).sum(1)
    ldo = (W + 127) // 64 * 64
    tol = dict(atol=2e-5, rtol=2e-5)
    rough = tol if hdt == F32 else dict(atol=0.03, rtol=1e-2)

    def run(**kw):
        out, hs, xo, save = torch.full((T, ldo), 7.0, device="cuda", dtype=hdt), torch.full((T, ldo), 7.0, device="cuda", dtype=hdt), r(T, W), r(6, W)
        kw = dict(x_out=xo, out=out, out_shift=hs, save=save, pos=pos, slot=slot, behind=behind, M=T, width=W, ldo=ldo, out_f32=int(hdt == F32), alpha=alpha, eps=eps) | kw
        kept = {k: v for k, v in kw.items() if v is not None}
        saved = save.clone()
        mo.post_norm(mo.PostNorm(**{k: v.data_ptr() if isinstance(v, torch.Tensor) else v for k, v in kept.items()}))
        return xo, out, hs, saved, save

    def previous(want):
        prev = torch.zeros_like(want)
        prev[1:] = want[:-1]
        first = torch.cat([torch.ones(1, dtype=torch.bool, device="cuda"), behind[:-1] == 0])
        prev[first] = torch.where((pos > 0)[:, None], before[slot.long()], torch.zeros((), device="cuda"))[first]
        return prev

    for kw, u in ((dict(y=y, ldy=W + 4), y[:T, :W]), (dict(y=y, ldy=W + 4, y_rows=place, y_top=2, y2=y2, ldy2=W + 8), picked + y2[:, :W])):
        for g in (None, gate):
            want = rms(alpha * x + (u if g is None else torch.sigmoid(g[:, :W] + b) * u), eps) * w
            gk = {} if g is None else dict(gate=gate, ldg=W + 12, gate_b=b)
            xo, out, hs, saved, save = run(x=x, w=w, shift=shift, before=before, **kw, **gk)
            assert torch.allclose(xo, want, **tol) and torch.allclose(out[:, :W].float(), want, **rough)
            assert torch.allclose(hs[:, :W].float(), want + (previous(want) - want) * shift, **rough)
            assert (out[:, W:] == 0).all() and (hs[:, W:] == 0).all()
            last = (behind == 0).nonzero()[:, 0]
            saved[slot[last].long()] = x[last]
            assert torch.equal(save, saved)
            rows = torch.tensor([T - 1, 2], dtype=torch.int32, device="cuda")
            res = run(x=x, w=w, rows=rows, M=2, w_out=wf, x_out=None, out_shift=None, save=None, **kw, **gk)[1]
            assert torch.allclose(res[:2, :W].float(), (rms(want, eps) * wf)[[T - 1, 2]], **rough) and (res[2:] == 7).all()
    # the first step
    tok, e = torch.randint(0, 50, (T,), dtype=torch.int32, device="cuda"), r(50, W).to(BF16)
    freq = torch.pow(torch.tensor(10000.0, dtype=torch.float64), -2.0 * torch.arange((W + 1) // 2, dtype=torch.float64) / W).cuda()
    far = pos + 3000
    a = far[:, None].double() * freq
    want = e[tok.long()].float() + torch.stack([a.sin(), a.cos()], -1).reshape(T, -1)[:, :W].float()
    xo, out, hs, _, _ = run(tokens=tok, embed=e, vocab=50, freq=freq, shift=shift, before=before, pos=far, save=None)
    first_seen = previous(want)
    first_seen[0] = before[slot[0].long()]                              # these positions have no first token
    at = [i for i in range(T) if i and behind[i - 1] == 0]
    first_seen[at] = before[slot[at].long()]
    assert torch.allclose(xo, want, **tol) and torch.allclose(hs[:, :W].float(), want + (first_seen - want) * shift, **rough)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M", [1, 3, 8, 40])
def test_one_product_with_two_inputs(M, dtype):
    from pocketllm_b200.models import mixer_layers as ml
    a, b = torch.randn(50, 100) * 0.1, torch.randn(37, 100) * 0.1
    f = ml.FusedLinear([("b", b)], dtype, "cuda", beside=[("a", a)])
    x, x2 = (torch.randn(M, f.K, device="cuda").to(dtype) for _ in range(2))
    ctx = ml.StepContext(M, *[None] * 6, ml.Workspace("cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"))
    y = f(ctx, x, "y", F32, beside=x2).double().cpu()
    xd, x2d = x[:, :100].double().cpu(), x2[:, :100].double().cpu()
    assert torch.allclose(y[:, :50], x2d @ a.to(dtype).double().t(), atol=1e-4) and torch.allclose(y[:, f.split:f.split + 37], xd @ b.to(dtype).double().t(), atol=1e-4)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,E,top,W,ff,shared", [(1, 5, 2, 72, 36, 50), (8, 3, 3, 130, 200, 20), (37, 7, 1, 72, 36, 130), (150, 4, 2, 264, 130, None), (3, 300, 5, 64, 20, 64),
                                                 (90, 70, 4, 64, 40, 300)])
def test_biased_router_and_shared_expert(T, E, top, W, ff, shared, dtype):
    """Both forms of the experts, a bias that is part of the logits, a shared expert; decisions are far apart and some hang on the bias."""
    from pocketllm_b200.models import mixer_layers as ml
    from pocketllm_b200.ops import mixer_ops as mo
    g = torch.Generator().manual_seed(T + E)
    r = lambda *s: torch.randn(*s, generator=g).to(BF16).float()
    x = r(T, W)
    gate, up, down = r(E, ff, W) * W ** -0.5, r(E, ff, W) * W ** -0.5, r(E, W, ff) * ff ** -0.5
    order = torch.stack([torch.randperm(E, generator=g) for _ in range(T)])
    bias = torch.zeros(E)
    bias[0] = 1.9                                                       # never the order's gap times a whole number
    sh = {"gate": r(shared, W) * W ** -0.5, "up": r(shared, W) * W ** -0.5, "down": r(W, shared) * shared ** -0.5} if shared else None
    m = ml.RoutedExperts(r(E, W) * 0.02, list(up), list(down), mo.Router(E, top, score="softmax", renorm=True, on_output=True), dtype, "cuda", gate=list(gate),
                         bias=bias, shared=ml.SwiGLU(sh, dtype, "cuda", name="_s") if shared else None, out_gate=r(W, W) * 0.1)
    z = torch.full((T, m.router.N), 50.0)
    z[:, :E].scatter_(1, order, 1.5 - 0.4 * torch.arange(E).float().repeat(T, 1))
    zc = z.cuda()
    m.router = lambda ctx, h, name, dt: zc
    ctx = ml.StepContext(T, *[None] * 6, ml.Workspace("cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"))
    h = torch.zeros(T, m.up.shape[2], device="cuda", dtype=dtype)
    h[:, :W] = x.to(dtype)
    out = m.forward(ctx, h)
    y = out["y"][:, :W].double().cpu()
    if "y_rows" in out:
        y = y[out["y_rows"].long().cpu()].sum(1)
    assert ("y2" in out) == bool(shared) and out["gate"].shape[1] >= W
    if shared:
        y = y + out["y2"][:, :W].double().cpu()
    swiglu = lambda v, a, b, c: c.to(dtype).double() @ (torch.nn.functional.silu(a.to(dtype).double() @ v) * (b.to(dtype).double() @ v))
    want = []
    for t in range(T):
        v, s = x[t].double(), z[t, :E].double() + bias.double()
        ids = s.topk(top).indices
        o = sum(p * swiglu(v, gate[e], up[e], down[e]) for e, p in zip(ids.tolist(), torch.softmax(s[ids], 0)))
        want.append(o + swiglu(v, sh["gate"], sh["up"], sh["down"]) if shared else o)
    want = torch.stack(want)
    assert ((y - want).norm() / want.norm()).item() < (1e-5 if dtype == F32 else 8e-3) and int(ctx.status) == 0


# ---- every mechanism alone ----

ALONE = {
    "scan": config([scan()]),
    "scan_one": config([scan(inner=1, state=1, rank=1, conv=1)]),
    "scan_odd": config([scan(inner=37, state=5, rank=3, conv=2)]),
    "scan_state4": config([scan(inner=40, state=4, rank=64, conv=3)]),
    "scan_state16": config([scan(inner=72, state=16, rank=16)]),
    "scan_state17": config([scan(inner=30, state=17, rank=9, conv=5)]),
    "scan_state24": config([scan(inner=136, state=24, rank=33)]),
    "scan_state64": config([scan(inner=24, state=64, rank=40)]),
    "scan_state100": config([scan(inner=20, state=100, rank=8, conv=9)]),
    "scan_state256": config([scan(inner=12, state=256, rank=70)]),
    "scan_state150": config([scan(inner=9, state=150, rank=5)]),
    "scan_wide": config([scan(inner=260, state=8, rank=100)], width=40),
    "scan_experts": config([scan(moe(experts=6, top=3))]),
    "latent": config([latent()]),
    "latent_one": config([latent(heads=1, dim=1, vdim=1, q_rank=1, kv_rank=1, scale=1.0)]),
    "latent_odd": config([latent(heads=5, dim=7, vdim=3, q_rank=9, kv_rank=13, scale=-0.4)]),
    "latent_64": config([latent(heads=2, dim=64, vdim=64, q_rank=64, kv_rank=64, scale=0.125)]),
    "latent_wide_values": config([latent(heads=2, dim=40, vdim=150, q_rank=100, kv_rank=70)]),
    "latent_wide_keys": config([latent(heads=2, dim=270, vdim=20, q_rank=24, kv_rank=30, scale=0.06)]),      # beyond the tensor-core form
    "latent_many_heads": config([latent(heads=19, dim=12, vdim=10, q_rank=50, kv_rank=130)]),
    "latent_steep": config([latent(scale=2.0)]),
    "latent_no_shared": config([latent(moe(shared=None))]),
    "forget": config([forget()]),
    "forget_one": config([forget(heads=1, dim=1, vdim=1)]),
    "forget_odd": config([forget(heads=3, dim=33, vdim=5)]),
    "forget_wide": config([forget(heads=2, dim=130, vdim=70)]),
    "forget_many": config([forget(heads=13, dim=6, vdim=128)]),
    "forget_experts": config([forget(moe(experts=1, top=1, ff=20, shared=200))], width=65),
    "alpha_small": config([forget(moe()), latent()], alpha=0.3),
    "alpha_negative": config([scan(moe()), forget()], alpha=-1.2),
    "width_odd": config([scan(moe()), latent(), forget()], width=71),
    "weights_shared": config([scan(moe()), again(scan(moe()), 0), latent(), forget(), again(latent(), 2), again(forget(), 3), again(scan(moe()), 1)]),
    "weights_from_behind": config([again(forget(moe()), 2), latent(), forget(moe())]),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(ALONE))
def test_mechanism_alone(name, dtype):
    cfg = ALONE[name]
    t = tensors(cfg, 3)
    if any(L["mlp"] for L in cfg["layers"]):
        t = clear_routes(cfg, t)
    seq = tokens(140, cfg["vocab"], 1)
    want = oracle(cfg, t, seq, "alone " + name)
    rt = runtime(cfg, t, dtype)
    check(feed(rt, "p", seq, [140]), want, dtype)
    check(feed(rt, "d", seq, [1]), want, dtype)
    check(feed(rt, "m", seq, [70, 1, 2, 9, 1, 64, 3]), want, dtype)


@pytest.mark.parametrize("kind", ["scan", "forget"])
@pytest.mark.parametrize("steps", ["fast", "slow"])
def test_memories_at_both_ends(kind, steps):
    """States that forget within a token, and states in which the first token still shows in the logits after hundreds."""
    cfg = config([scan() if kind == "scan" else forget()])
    t = tensors(cfg, 4)
    fast, full = steps == "fast", lambda n, v: torch.full_like(t["l0.mix." + n], v)
    if kind == "scan":
        t.update({"l0.mix.A_log": full("A_log", 4.0 if fast else -6.0), "l0.mix.dt.b": full("dt.b", 3.0 if fast else -1.0)})
    else:
        t.update({"l0.mix.f.b": full("f.b", -9.0 if fast else 8.0), "l0.mix.lower": full("lower", 0.0 if fast else 0.75)})
    t["l0.mix.o"] = (t["l0.mix.o"].float() * 3).to(BF16)
    seq = tokens(400, cfg["vocab"], 8)
    want = zr.PlainModel(cfg, t).logits(seq)
    if not fast:
        other = zr.PlainModel(cfg, t).logits([(seq[0] + 1) % 83] + seq[1:])
        assert ((want - other).pow(2).mean(-1).sqrt() / want.std())[390] > 1e-3
    # a state that is all this token's value leaves the head norm little but the sign of the query's sum, which 16 bits can turn
    for dtype in (F32, BF16) if kind == "scan" or not fast else (F32,):
        rt = runtime(cfg, t, dtype)
        check(feed(rt, "a", seq, [400]), want, dtype)
        check(feed(rt, "a", seq, [200, 1, 130, 1]), want, dtype)


@pytest.mark.parametrize("lower", [0.0, 1.0])
def test_bounds_of_the_forget_gate(lower):
    """A gate without a bound, far into both of its ends, and one that never forgets and never writes (the outputs are then zero)."""
    cfg = config([forget()])
    t = tensors(cfg, 5)
    t["l0.mix.lower"] = torch.full_like(t["l0.mix.lower"], lower)
    t["l0.mix.f.b"] = torch.linspace(-60.0, 60.0, 100).to(BF16)
    seq = tokens(150, cfg["vocab"], 9)
    want = oracle(cfg, t, seq, f"lower {lower}")
    for dtype in (F32, BF16):
        rt = runtime(cfg, t, dtype)
        for cuts in ([150], [1], [9, 64, 2]):
            check(feed(rt, "a", seq, cuts), want, dtype)


@pytest.mark.parametrize("taps", [2, 4, 5])
def test_convolution_and_shift_at_portion_edges(taps):
    """The line of the convolution and the previous token's input over portions shorter and longer than the line, in a slot that another
    request has left."""
    cfg = config([scan(conv=taps), scan(moe(), inner=20, conv=taps + 1)])
    t = clear_routes(cfg, tensors(cfg, 6))
    t["l0.shift"], t["l1.shift"] = torch.ones_like(t["l0.shift"]), torch.full_like(t["l1.shift"], 0.5)
    rt = runtime(cfg, t, max_requests=1, pages=3)
    for k, cuts in enumerate(([1], [2], [3, 1, 2], [9, 1, 10, 2], [64, 2, 9], [65, 1, 1, 1, 12])):
        seq = tokens(110, cfg["vocab"], 40 + k)
        check(feed(rt, k, seq, cuts), oracle(cfg, t, seq, f"taps {taps} {k}"))


# ---- the whole design ----

def full_tensors(seed):
    return clear_routes(FULL, tensors(FULL, seed))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cuts", [[200], [1], [2], [7], [9], [63, 65, 2], [64], [128, 3, 1, 1, 50], [199, 1]])
def test_portions(cuts, dtype):
    t = full_tensors(7)
    seq = tokens(200, FULL["vocab"], 2)
    want = oracle(FULL, t, seq, "full")
    check(feed(runtime(FULL, t, dtype), "r", seq, cuts), want, dtype)


def test_random_routers_in_fp32():
    """Routers whose decisions are as close as chance makes them."""
    t = tensors(FULL, 9)
    seq = tokens(120, FULL["vocab"], 4)
    want = zr.PlainModel(FULL, t).logits(seq)
    rt = runtime(FULL, t)
    check(feed(rt, "a", seq, [120]), want)
    check(feed(rt, "a", seq, [50, 1, 8, 40]), want)


def test_layers_one_by_one():
    """The residual stream behind every layer, in prompts and single tokens; the logits do not depend on who looks."""
    from pocketllm_b200.runtime.mixer_runtime import StepEntry
    t = full_tensors(2)
    seq = tokens(30, FULL["vocab"], 4)
    m = zr.PlainModel(FULL, t)
    st, want = m.new_state(), []
    for k in seq:
        row = []
        m.step(st, k, row)
        want.append(torch.stack(row))
    want = torch.stack(want, 1)
    for dtype in (F32, BF16):
        rt = runtime(FULL, t, dtype)
        rt.launch_layers = []
        for a, b in ((0, 26), (26, 27), (27, 30)):
            z = rt.step([StepEntry("a", seq[a:b], (b - a - 1,))]).double().cpu()
        n = len(FULL["layers"])
        got = [torch.cat(rt.launch_layers[i::n]).double().cpu() for i in range(n)]
        for i in range(n):
            assert ((got[i] - want[i]).norm() / want[i].norm()).item() < (3e-6 if dtype == F32 else 2e-2)
        plain = feed(runtime(FULL, t, dtype), "b", seq, [26, 1, 3])[-1:]
        assert ((plain - z).norm() / z.norm()).item() < (1e-6 if dtype == F32 else 1e-3)


def test_logits_of_some_places_and_of_none():
    from pocketllm_b200.runtime.mixer_runtime import StepEntry
    for cfg in (FULL, config([scan(), forget()])):                       # the second ends without a feed-forward
        t = clear_routes(cfg, tensors(cfg, 14))
        seq = tokens(60, cfg["vocab"], 5)
        want = zr.PlainModel(cfg, t).logits(seq)
        rt = runtime(cfg, t)
        assert rt.step([StepEntry("a", seq[:20])]).shape == (0, cfg["vocab"])
        z = rt.step([StepEntry("a", seq[20:45], (24, 0, 7)), StepEntry("b", seq[:3], (1,))]).double().cpu()
        check(z, torch.cat([want[[44, 20, 27]], want[[1]]]))
        rt.step([StepEntry("a", seq[45:46])])
        check(rt.step([StepEntry("a", seq[46:47], (0,))]).double().cpu(), want[[46]])


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_requests_in_one_batch_and_reused_room(dtype):
    """Nine requests through three slots and few pages. Every place is compared with the request alone."""
    t = full_tensors(8)
    seqs = [tokens(n, FULL["vocab"], 20 + i) for i, n in enumerate([150, 1, 65, 64, 2, 77, 128, 33, 17])]
    got = traffic(runtime(FULL, t, dtype, max_requests=3, pages=7), seqs, 3, 7)
    for i, (seq, z) in enumerate(zip(seqs, got)):
        check(z, oracle(FULL, t, seq, f"traffic {i}"), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_decode_batches(dtype):
    """Single tokens of several requests together, twice per batch size so that the captured graph runs, against each alone."""
    from pocketllm_b200.runtime.mixer_runtime import StepEntry
    t = full_tensors(8)
    seqs = [tokens(40 + 9 * i, FULL["vocab"], 70 + i) for i in range(4)]
    rt = runtime(FULL, t, dtype)
    for i, s in enumerate(seqs):
        rt.step([StepEntry(i, s[:-20])])
    got = {i: [] for i in range(4)}
    for k in range(20):
        who = [i for i in range(4) if (k + i) % 5]
        z = rt.step([StepEntry(i, [seqs[i][len(seqs[i]) - 20 + len(got[i])]], (0,)) for i in who]).double().cpu()
        for i, row in zip(who, z):
            got[i].append(row)
    rt.check_status()
    for i, s in enumerate(seqs):
        n = len(got[i])
        check(torch.stack(got[i]), oracle(FULL, t, s, f"decode {i}")[len(s) - 20:len(s) - 20 + n], dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_many_short_portions_in_one_batch(dtype):
    """Seven requests whose portions of one to eight tokens share blocks of the scan, some of them resting."""
    from pocketllm_b200.runtime.mixer_runtime import StepEntry
    cfg = config([scan(), forget(), scan(inner=45, state=33, rank=50)])
    t = tensors(cfg, 15)
    seqs = [tokens(30 + 3 * i, cfg["vocab"], 110 + i) for i in range(7)]
    rt = runtime(cfg, t, dtype, max_requests=7, pages=7)
    at, got, k = [0] * 7, [[] for _ in seqs], 0
    while any(a < len(s) for a, s in zip(at, seqs)):
        e = [StepEntry(i, s[at[i]:at[i] + 1 + (3 * i + 5 * k) % 8], ()) for i, s in enumerate(seqs) if at[i] < len(s) and (i + k) % 4]
        k += 1
        for x in e:
            x.want = range(len(x.tokens))
        z = rt.step(e).double().cpu() if e else []
        for x in e:
            n = len(x.tokens)
            got[x.rid].append(z[:n])
            z = z[n:]
            at[x.rid] += n
    rt.check_status()
    for i, s in enumerate(seqs):
        check(torch.cat(got[i]), oracle(cfg, t, s, f"short {i}"), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_one_key_at_page_borders(dtype):
    """One key stands out: at page borders, at the start of the sequence and far back, in prompts, short portions and single tokens."""
    cfg = config([latent(), latent(heads=1, dim=4, vdim=13)])
    t = beacon_tensors(cfg)
    m = zr.PlainModel(cfg, t)
    rt = runtime(cfg, t, dtype)
    for place in (0, 20, 63, 64, 127):
        seq = tokens(145, cfg["vocab"], 30 + place, low=1)
        seq[place] = BEACON
        want = m.logits(seq)
        check(feed(rt, "p", seq, [145]), want, dtype)
        check(feed(rt, "d", seq, [max(1, place - 3), 1]), want, dtype)
        check(feed(rt, "s", seq, [place + 7, 2, 2, 2, 8]), want, dtype)
        check(feed(rt, "c", seq, [place + 11, 33]), want, dtype)


def test_first_tokens():
    t = full_tensors(5)
    for n in (1, 2, 3):
        seq = tokens(n, FULL["vocab"], 90 + n)
        want = zr.PlainModel(FULL, t).logits(seq)
        for dtype in (F32, BF16):
            rt = runtime(FULL, t, dtype)
            check(feed(rt, "a", seq, [n]), want, dtype)
            check(feed(rt, "a", seq, [1]), want, dtype)


def test_split_context_decode():
    """Context long enough for several splits of the row kernel, with a far key that stands out."""
    cfg = config([latent()])
    t = beacon_tensors(cfg)
    seq = tokens(600, cfg["vocab"], 77, low=1)
    seq[37] = BEACON
    want = zr.PlainModel(cfg, t).logits(seq)
    for dtype in (F32, BF16):
        rt = runtime(cfg, t, dtype, pages=24)
        assert rt.model.layers[0].mixer.nsplit > 4
        check(feed(rt, "a", seq, [590, 1]), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """280 single tokens after a short prompt, through graphs, over several pages."""
    t = full_tensors(11)
    seq = tokens(300, FULL["vocab"], 6)
    want = oracle(FULL, t, seq, "long")
    check(feed(runtime(FULL, t, dtype), "a", seq, [20, 1]), want, dtype)


def test_greedy_generation_through_the_scheduler():
    from pocketllm_b200.runtime.batching import BatchEngine
    from pocketllm_b200.server.backends import MixerBackend
    from pocketllm_b200.server.engine import ServingEngine
    t = full_tensors(12)
    m = zr.PlainModel(FULL, t)
    prompts = [tokens(n, FULL["vocab"], 60 + n) for n in (3, 90, 1, 40, 66)]
    lens = [30, 12, 40, 9, 20]
    rt = runtime(FULL, t, max_requests=3, pages=6)
    eng = BatchEngine(rt, token_budget=64)
    outs = eng.run(prompts, [SamplingParams(max_tokens=n) for n in lens])
    for p, o, n in zip(prompts, outs, lens):
        ref = margin_prefix(m, p, n, 1e-4)
        assert len(o) == n and len(ref) > min(n, 4) and o[:len(ref)] == ref
    assert eng.stats["burst_steps"] > 0 and eng.stats["mixed_steps"] > 0 and rt.cache.free_pages == 6
    # the single-request interface and the server's engine
    rt.reset()
    first = rt.prefill(prompts[1], portion=33)
    assert [first] + [first := rt.decode_one(first) for _ in range(5)] == outs[1][:6]
    rt.reset()
    srv = ServingEngine(MixerBackend(rt))
    got = [int(x) for x in srv.stream(prompts[3], SamplingParams(max_tokens=9)) if not isinstance(x, tuple)]
    srv.close()
    assert got == outs[3]


def test_command_line_and_trace_runner(tmp_path):
    """The generation CLI and bin/trace_run on a checkpoint folder: generation's tokens are the arg-max of the replayed logits."""
    t = full_tensors(13)
    zx.save_checkpoint(tmp_path / "m", zx.ZarinexConfig.from_dict(FULL), t)
    ids = [ord(c) % 101 for c in "Qy7 =b"]
    r = subprocess.run([sys.executable, "-m", "pocketllm_b200.cli.generate", "--ckpt-path", str(tmp_path / "m"), "--tokenizer-path", "chars", "--prompt",
                        "".join(chr(i) for i in ids), "--max-new-tokens", "6", "--max-context", "256", "--dtype", "float32"],
                       cwd=ROOT, capture_output=True, timeout=280)
    assert r.returncode == 0, r.stderr.decode()
    want = zr.PlainModel(FULL, t).generate(ids, 6)
    assert r.stdout.decode() == "".join(chr(i) for i in want) + "\n"
    seq = tokens(70, 101, 3)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seq[:40], "want": [39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": seq[40:41], "want": []}, {"id": "b", "tokens": seq[:30], "want": [0, 29]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": seq[30:31], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": seq, "want": [69]}], "end": ["c"]}]
    ref = zr.PlainModel(FULL, t).logits(seq)
    for dt in ("float32", "bfloat16"):
        out = tmp_path / dt
        out.mkdir()
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dt, "--out", str(out), "--max-tokens", "128"],
                           input="".join(json.dumps(s) + "\n" for s in steps).encode(), capture_output=True, timeout=280)
        assert r.returncode == 0, r.stderr.decode()
        assert [x for x in r.stdout.decode().split("\n") if x.startswith("done")] == [f"done {i}" for i in range(4)]
        for s, places in ((0, [39]), (1, [0, 29]), (2, [30]), (3, [69])):
            z = torch.frombuffer(bytearray((out / f"{s}.f32").read_bytes()), dtype=torch.float32).view(-1, 101).double()
            check(z, ref[places], getattr(torch, dt))
