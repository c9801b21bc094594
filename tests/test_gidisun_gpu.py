"""Gidisun on the GPU against the plain oracle (float64, token by token): every mechanism alone, prompts, portions, mixed
batches, reused pages and slots, windows' edges, long decoding, unusual sizes, generation through the scheduler, the CLI."""
import json
import subprocess
import sys
from pathlib import Path

import mixer_reference as mr
import pytest
import torch
from gidisun_cases import BEACON, beacon_tensors, config, gla, latent, mlstm, tensors, tokens
from mixer_checks import BF16, F32, check, feed, make_runtime, margin_prefix, traffic

from pocketllm_b200.models import gidisun as gd
from pocketllm_b200.server.engine import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
FULL = config([mlstm(ff=90), latent(ff=70), gla(), latent(heads=2, window=17, scaling=False), mlstm(heads=1, dim=9, vdim=40)], vocab=101, width=88)


def runtime(cfg, t, dtype=F32, **kw):
    return make_runtime(gd, gd.GidisunConfig, cfg, t, dtype, **kw)


_memo: dict = {}


def oracle(cfg, t, seq, key):
    k = (key, len(seq))
    if k not in _memo:
        _memo[k] = mr.PlainModel(cfg, t).logits(seq)
    return _memo[k]


# ---- kernels ----

@pytest.mark.parametrize("M,N,K", [(1, 40, 64), (3, 33, 128), (8, 257, 1024), (2, 4096, 2048), (5, 8, 4160)])
def test_linear_rows(M, N, K):
    from pocketllm_b200.ops import mixer_ops as mo
    g = torch.Generator(device="cuda").manual_seed(N)
    x = torch.randn(M, K, generator=g, device="cuda").to(BF16)
    w = (torch.randn(N, K, generator=g, device="cuda") * K ** -0.5).to(BF16)
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    ref = x.float() @ w.float().t()
    for dt, tol in ((F32, 1e-5), (BF16, 5e-3)):
        y = mo.linear(x, w, torch.empty(M, N, device="cuda", dtype=dt), st)
        assert ((y.float() - ref).norm() / ref.norm()).item() < tol
    if N % 2 == 0:
        y = mo.linear(x, w, torch.empty(M, N // 2, device="cuda", dtype=BF16), st, swiglu=True)
        r = torch.nn.functional.silu(ref[:, :N // 2]) * ref[:, N // 2:]
        assert ((y.float() - r).norm() / r.norm()).item() < 5e-3


@pytest.mark.parametrize("M,N,K", [(1, 40, 64), (4, 30, 100), (7, 66, 33), (70, 130, 90), (129, 64, 256)])
def test_linear_f32(M, N, K):
    from pocketllm_b200.ops import mixer_ops as mo
    x, w = torch.randn(M, K, device="cuda"), torch.randn(N, K, device="cuda") * K ** -0.5
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    ref = x.double() @ w.double().t()
    y = mo.linear(x, w, torch.empty(M, N, device="cuda"), st)
    assert ((y - ref).norm() / ref.norm()).item() < 1e-6
    y = mo.linear(x, w, torch.empty(M, N // 2, device="cuda"), st, swiglu=True)
    r = torch.nn.functional.silu(ref[:, :N // 2]) * ref[:, N // 2:]
    assert ((y - r).norm() / r.norm()).item() < 1e-6


@pytest.mark.parametrize("W", [24, 300, 2048, 5000])
@pytest.mark.parametrize("plus_one", [True, False])
def test_sandwich_norm(W, plus_one):
    from pocketllm_b200.ops import mixer_ops as mo
    T, V, eps, b = 6, 11, 1e-3, 1.0 if plus_one else 0.0
    x, y = torch.randn(T, W, device="cuda"), torch.randn(T, W + 8, device="cuda")
    wp, wn = torch.randn(W, device="cuda"), torch.randn(W, device="cuda")
    rms = lambda v: v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)
    want_x = x + rms(y[:, :W]) * (b + wp)
    out = torch.full((T, W + 16), 7.0, device="cuda")
    x2 = x.clone()
    mo.sandwich_norm(x2, y=y, w_post=wp, w_pre=wn, out=out, eps=eps, plus_one=plus_one)
    assert torch.allclose(x2, want_x, atol=1e-5) and torch.allclose(out[:, :W], rms(want_x) * (b + wn), atol=1e-4, rtol=1e-4)
    assert (out[:, W:] == 0).all()
    rows = torch.tensor([4, 1], dtype=torch.int32, device="cuda")
    o2 = torch.empty(2, W, device="cuda", dtype=BF16)
    x3 = x.clone()
    mo.sandwich_norm(x3, y=y, w_post=wp, rows=rows, w_pre=wn, out=o2, eps=eps, plus_one=plus_one)
    assert torch.equal(x3, x) and torch.allclose(o2.float(), (rms(want_x) * (b + wn))[[4, 1]], atol=0.05, rtol=0.02)
    emb = torch.randn(V, W, device="cuda").to(BF16)
    toks = torch.tensor([0, 3, V - 1, 5, 5, 1], dtype=torch.int32, device="cuda")
    mo.sandwich_norm(x3, tokens=toks, embed=emb, w_pre=wn, out=out, eps=eps, plus_one=plus_one)
    assert torch.equal(x3, emb[toks.long()].float()) and torch.allclose(out[:, :W], rms(x3) * (b + wn), atol=1e-4, rtol=1e-4)


# ---- every mechanism alone ----

ALONE = {
    "mlstm": config([mlstm()]),
    "mlstm_wide": config([mlstm(heads=2, dim=70, vdim=33, cap=2.0)]),
    "mlstm_one": config([mlstm(heads=1, dim=1, vdim=1)]),
    "mlstm_big": config([mlstm(heads=1, dim=260, vdim=140)], width=64),
    "gla": config([gla()]),
    "gla_wide": config([gla(heads=1, dim=130, vdim=70, tau=1.0)]),
    "gla_one": config([gla(heads=2, dim=1, vdim=1, tau=16.0)]),
    "latent": config([latent()]),
    "latent_full": config([latent(window=None, scaling=False)]),
    "latent_window1": config([latent(window=1)]),
    "latent_one": config([latent(heads=1, dim=2, rot=2, vdim=5, rank=3, window=5, scale=1.0)]),
    "latent_values": config([latent(heads=2, dim=60, rot=20, vdim=150, rank=200, window=70)]),        # several value slices
    "latent_wide_keys": config([latent(heads=2, dim=250, rot=16, vdim=20, rank=50, window=33)]),       # keys beyond the tensor-core form
    "latent_rank": config([latent(heads=9, dim=8, rot=8, vdim=16, rank=600, window=100)]),             # more than one column pair per thread
    "swiglu": config([gla(ff=130)], width=65),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(ALONE))
def test_mechanism_alone(name, dtype):
    cfg = ALONE[name]
    t = tensors(cfg, 3)
    seq = tokens(150, cfg["vocab"], 1)
    want = oracle(cfg, t, seq, "alone " + name)
    rt = runtime(cfg, t, dtype)
    got = feed(rt, "p", seq, [150])
    check(got, want, dtype)
    check(feed(rt, "d", seq, [1]), want, dtype)
    check(feed(rt, "m", seq, [70, 1, 2, 9, 1, 64, 3]), want, dtype)


@pytest.mark.parametrize("tau,bias", [(1.0, -6.0), (16.0, 8.0), (1.0, 30.0)])
def test_extreme_decays(tau, bias):
    """Decays close to 0 and to 1: neither the chunk form nor its sub-chunks may overflow or lose the state."""
    cfg = config([gla(tau=tau)])
    t = tensors(cfg, 5)
    t["l0.mix.a2.b"] = (bias + 3.0 * torch.randn(t["l0.mix.a2.b"].shape, generator=torch.Generator().manual_seed(1))).to(BF16)
    seq = tokens(200, cfg["vocab"], 4)
    want = mr.PlainModel(cfg, t).logits(seq)
    rt = runtime(cfg, t)
    check(feed(rt, "a", seq, [200]), want)
    check(feed(rt, "a", seq, [1]), want)


@pytest.mark.parametrize("fb,ib", [(-8.0, 0.0), (9.0, 4.0), (9.0, -9.0), (0.0, -12.0)])
def test_extreme_gates(fb, ib):
    """Forget gates near 0 and 1, input gates at both ends of the cap: the running maximum, its start at 0 and the lower
    bound of the denominator all matter."""
    cfg = config([mlstm(cap=11.0)])
    t = tensors(cfg, 6)
    for n, b in (("f", fb), ("i", ib)):
        t[f"l0.mix.{n}.b"] = (b + torch.randn(3, generator=torch.Generator().manual_seed(2))).to(BF16)
        t[f"l0.mix.{n}"] = (t[f"l0.mix.{n}"].float() * 4).to(BF16)
    seq = tokens(330, cfg["vocab"], 4)
    want = mr.PlainModel(cfg, t).logits(seq)
    rt = runtime(cfg, t)
    check(feed(rt, "a", seq, [330]), want, factor=3)
    check(feed(rt, "a", seq, [300, 1]), want, factor=3)


# ---- the whole design ----

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cuts", [[300], [1], [2], [7], [9], [63, 65, 2], [64], [128, 3, 1, 1, 100], [299, 1]])
def test_portions(cuts, dtype):
    t = tensors(FULL, 7)
    seq = tokens(300, FULL["vocab"], 2)
    want = oracle(FULL, t, seq, "full")
    check(feed(runtime(FULL, t, dtype), "r", seq, cuts), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_requests_in_one_batch_and_reused_room(dtype):
    """Twelve requests through three slots and few pages. Every place is compared with the request alone."""
    t = tensors(FULL, 8)
    seqs = [tokens(n, FULL["vocab"], 20 + i) for i, n in enumerate([200, 1, 65, 64, 130, 2, 77, 9, 128, 33, 190, 17])]
    got = traffic(runtime(FULL, t, dtype, max_requests=3, pages=9), seqs, 3, 9)
    m = mr.PlainModel(FULL, t)
    for seq, z in zip(seqs, got):
        check(z, m.logits(seq), dtype)


def test_wanted_places_and_errors():
    from pocketllm_b200.runtime.mixer_runtime import StepEntry
    from pocketllm_b200.runtime.request_cache import CacheFull
    t = tensors(FULL, 7)
    seq = tokens(300, FULL["vocab"], 2)
    want = oracle(FULL, t, seq, "full")
    rt = runtime(FULL, t, max_requests=2, pages=6)
    assert rt.step([StepEntry("a", seq[:20])]).shape == (0, FULL["vocab"])
    z = rt.step([StepEntry("a", seq[20:60], (39, 3)), StepEntry("b", seq[:11], (10,))]).double().cpu()
    check(z, want[[59, 23, 10]])
    z = rt.step([StepEntry("b", seq[11:12]), StepEntry("a", seq[60:61], (0,))]).double().cpu()
    check(z, want[[60]])
    for bad in ([StepEntry("a", [])], [StepEntry("a", [FULL["vocab"]])], [StepEntry("a", [1], (1,))], [StepEntry("a", [1]), StepEntry("a", [1])]):
        with pytest.raises(ValueError):
            rt.step(bad)
    for bad in ([StepEntry("c", [1])], [StepEntry("a", seq[61:300] + [1] * 140)]):
        with pytest.raises(CacheFull):
            rt.step(bad)
    check(rt.step([StepEntry("a", seq[61:100], (38,))]).double().cpu(), want[[99]])     # nothing was disturbed


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [29, 64, 65, None])
def test_keys_at_window_and_page_edges(window, dtype):
    """One key stands out: seen up to the window's last position and not one later, at page borders, at the start of the
    sequence and far back; in prompts, short portions and single tokens."""
    cfg = config([latent(window=window), gla(heads=1, dim=4, vdim=6)])
    t = beacon_tensors(cfg)
    m = mr.PlainModel(cfg, t)
    rt = runtime(cfg, t, dtype)
    for place in (0, 20, 63, 64):
        seq = tokens(140, cfg["vocab"], 30 + place, low=1)
        seq[place] = BEACON
        want = m.logits(seq)
        check(feed(rt, "p", seq, [140]), want, dtype)
        check(feed(rt, "d", seq, [place + 20, 1]), want, dtype)
        check(feed(rt, "s", seq, [place + 27 if place else 5, 2, 2, 2, 8]), want, dtype)
        check(feed(rt, "c", seq, [place + 11, 33]), want, dtype)


def test_sinks_and_first_tokens():
    cfg = config([latent(heads=4, window=40)])
    t = beacon_tensors(cfg)
    seq = tokens(12, cfg["vocab"], 9, low=1)
    want = mr.PlainModel(cfg, t).logits(seq)
    for dtype in (F32, BF16):
        rt = runtime(cfg, t, dtype)
        for cuts in ([12], [1], [9, 1], [2]):
            check(feed(rt, "a", seq, cuts), want, dtype)
    t2 = dict(t)
    t2["l0.mix.sink"] = torch.full((4,), -60.0, dtype=BF16)          # a sink nobody notices: the other branch of the merge
    check(feed(runtime(cfg, t2), "a", seq, [4, 1]), mr.PlainModel(cfg, t2).logits(seq))


def test_split_context_decode():
    """Context long enough for several splits of the row kernel, with a far key that stands out."""
    cfg = config([latent(window=None, heads=3)])
    t = beacon_tensors(cfg)
    seq = tokens(700, cfg["vocab"], 77, low=1)
    seq[37] = BEACON
    want = mr.PlainModel(cfg, t).logits(seq[:700])
    for dtype in (F32, BF16):
        rt = runtime(cfg, t, dtype, pages=24)
        assert rt.model.layers[0].mixer.nsplit > 4
        got = feed(rt, "a", seq, [690, 1])
        check(got, want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """400 single tokens after a short prompt, through graphs and the device feedback, over several pages."""
    t = tensors(FULL, 11)
    seq = tokens(420, FULL["vocab"], 6)
    want = oracle(FULL, t, seq, "long")
    rt = runtime(FULL, t, dtype)
    check(feed(rt, "a", seq, [20, 1]), want, dtype)


def test_greedy_generation_through_the_scheduler():
    from pocketllm_b200.runtime.batching import BatchEngine
    t = tensors(FULL, 12)
    m = mr.PlainModel(FULL, t)
    prompts = [tokens(n, FULL["vocab"], 60 + n) for n in (3, 90, 1, 40, 66, 12, 150)]
    lens = [40, 20, 70, 9, 30, 64, 5]
    rt = runtime(FULL, t, max_requests=3, pages=8)
    eng = BatchEngine(rt, token_budget=64)
    outs = eng.run(prompts, [SamplingParams(max_tokens=n) for n in lens])
    for p, o, n in zip(prompts, outs, lens):
        ref = margin_prefix(m, p, n, 1e-4)
        assert len(o) == n and len(ref) > min(n, 4) and o[:len(ref)] == ref
    assert eng.stats["burst_steps"] > 0 and eng.stats["mixed_steps"] > 0 and rt.cache.free_pages == 8
    alone = [BatchEngine(runtime(FULL, t, max_requests=1, pages=8, use_graphs=False), burst=1).run([p], [SamplingParams(max_tokens=n)])[0]
             for p, n in list(zip(prompts, lens))[:3]]
    for p, o, a in zip(prompts, outs, alone):
        k = len(margin_prefix(m, p, len(o), 1e-4))
        assert o[:k] == a[:k]
    # the single-request interface and the server's engine
    rt.reset()
    first = rt.prefill(prompts[1], portion=33)
    assert [first] + [first := rt.decode_one(first) for _ in range(5)] == outs[1][:6]
    rt.reset()
    from pocketllm_b200.server.backends import MixerBackend
    from pocketllm_b200.server.engine import ServingEngine
    srv = ServingEngine(MixerBackend(rt))
    got = [int(x) for x in srv.stream(prompts[3], SamplingParams(max_tokens=9)) if not isinstance(x, tuple)]
    srv.close()
    assert got == outs[3]


def test_command_line_and_trace_runner(tmp_path):
    """The generation CLI and bin/trace_run on a checkpoint folder: generation's tokens are the arg-max of the replayed logits."""
    t = tensors(FULL, 13)
    gd.save_checkpoint(tmp_path / "m", gd.GidisunConfig.from_dict(FULL), t)
    prompt = "Za4 _x"
    r = subprocess.run([sys.executable, "-m", "pocketllm_b200.cli.generate", "--ckpt-path", str(tmp_path / "m"), "--tokenizer-path", "chars", "--prompt",
                        "".join(chr(ord(c) % 101) for c in prompt), "--max-new-tokens", "6", "--max-context", "256", "--dtype", "float32"],
                       cwd=ROOT, capture_output=True, timeout=280)
    assert r.returncode == 0, r.stderr.decode()
    ids = [ord(c) % 101 for c in prompt]
    want = mr.PlainModel(FULL, t).generate(ids, 6)
    assert r.stdout.decode() == "".join(chr(i) for i in want) + "\n"
    seq = tokens(70, 101, 3)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seq[:40], "want": [39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": seq[40:41], "want": []}, {"id": "b", "tokens": seq[:30], "want": [0, 29]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": seq[30:31], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": seq, "want": [69]}], "end": ["c"]}]
    for dt in ("float32", "bfloat16"):
        out = tmp_path / dt
        out.mkdir()
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dt, "--out", str(out), "--max-tokens", "128"],
                           input="".join(json.dumps(s) + "\n" for s in steps).encode(), capture_output=True, timeout=280)
        assert r.returncode == 0, r.stderr.decode()
        assert [x for x in r.stdout.decode().split("\n") if x.startswith("done")] == [f"done {i}" for i in range(4)]
        ref = mr.PlainModel(FULL, t).logits(seq)
        for s, places in ((0, [39]), (1, [0, 29]), (2, [30]), (3, [69])):
            z = torch.frombuffer(bytearray((out / f"{s}.f32").read_bytes()), dtype=torch.float32).view(-1, 101).double()
            check(z, ref[places], getattr(torch, dt))
