"""Zemozen on the GPU against the plain oracle (float64, token by token): every mechanism alone, prompts, portions, mixed
batches, reused pages and slots, window edges, long decoding, unusual sizes, generation through the scheduler, the CLI."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch
import zemozen_reference as zr
from mixer_checks import BF16, F32, check, feed, make_runtime, margin_prefix, traffic
from mixer_reference import rms
from zemozen_cases import BEACON, FULL, attention, beacon_tensors, clear_routes, config, moe, parallel, tensors, tokens

from pocketllm_b200.models import zemozen as zm
from pocketllm_b200.server.engine import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def runtime(cfg, t, dtype=F32, **kw):
    return make_runtime(zm, zm.ZemozenConfig, cfg, t, dtype, **kw)


_memo: dict = {}


def oracle(cfg, t, seq, key):
    k = (key, len(seq))
    if k not in _memo:
        _memo[k] = zr.PlainModel(cfg, t).logits(seq)
    return _memo[k]


# ---- kernels ----

@pytest.mark.parametrize("hdt", [F32, BF16])
@pytest.mark.parametrize("W", [24, 301, 2048])
def test_residual_steps_with_factor_and_identities(W, hdt):
    """Sublayer outputs times a constant, missing expert rows, a row of the sublayer's input times a factor per token; the output
    may go where that input lies."""
    from pocketllm_b200.ops import mixer_ops as mo
    T, eps = 6, 1e-3
    x, y, wn = torch.randn(T, W, device="cuda"), torch.randn(2 * T, W + 4, device="cuda"), torch.randn(W, device="cuda")
    h = torch.randn(T, (W + 71) // 64 * 64, device="cuda").to(hdt)
    sw = torch.tensor([0.0, 0.7, 1.0, -0.4, 0.0, 2.0], device="cuda")
    place = torch.tensor([[0, 5], [-1, 3], [-1, -1], [11, -1], [2, 2], [7, -1]], dtype=torch.int32, device="cuda")
    picked = torch.where((place >= 0)[..., None], y[place.clamp(min=0).long(), :W], torch.zeros((), device="cuda")).sum(1)
    kw = dict(eps=eps, plus_one=False, y_scale=0.3, skip=h, skip_w=sw)
    for step, base in ((dict(y=y[:T]), y[:T, :W]), (dict(y=y, y_rows=place), picked)):
        want = x + 0.3 * (base + sw[:, None] * h[:, :W].float())
        for out in (torch.full_like(h, 7.0), None):
            a, hh = x.clone(), h.clone()
            dst = hh if out is None else out
            mo.sandwich_norm(a, w_pre=wn, out=dst, **step, **{**kw, "skip": hh})
            assert torch.allclose(a, want, atol=1e-5)
            assert torch.allclose(dst[:, :W].float(), rms(want, eps) * wn, atol=1e-4 if hdt == F32 else 0.05, rtol=1e-4 if hdt == F32 else 1e-2)
            assert (dst[:, W:] == 0).all()
        rows = torch.tensor([5, 1], dtype=torch.int32, device="cuda")
        out = torch.zeros(2, h.shape[1], device="cuda", dtype=F32)
        mo.sandwich_norm(x, rows=rows, count=2, w_pre=wn, out=out, **step, **kw)
        assert torch.allclose(out[:, :W], (rms(want, eps) * wn)[[5, 1]], atol=1e-4, rtol=1e-4)


def plain_experts(z, x, gate, up, down, top, corr, renorm, on_output, score):
    E, n = len(up), z.shape[1]
    s = torch.sigmoid(z) if score == "sigmoid" else torch.softmax(z, -1)
    ids = (s + corr).topk(top, -1).indices
    w = s.gather(1, ids)
    if renorm:
        w = w / w.sum(-1, keepdim=True)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(top):
            e, f = int(ids[t, j]), w[t, j]
            if e >= E:
                y[t] += f * x[t]
                continue
            v = x[t] if on_output else f * x[t]
            o = down[e] @ (torch.nn.functional.silu(gate[e] @ v) * (up[e] @ v))
            y[t] += f * o if on_output else o
    assert n >= E
    return y


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,E,ident,top,W,ff,kw", [
    (1, 5, 2, 2, 72, 36, {}), (8, 3, 1, 4, 130, 200, {}), (37, 7, 0, 3, 72, 36, {}), (150, 4, 4, 6, 264, 130, {}), (300, 90, 10, 2, 64, 128, {}),
    (3, 500, 12, 32, 64, 20, {}), (20, 1, 2, 1, 48, 40, {}), (5, 1, 1, 2, 48, 40, {}), (40, 9, 3, 2, 72, 50, dict(on_output=False)),
    (4, 9, 3, 2, 72, 50, dict(on_output=False, renorm=False)), (30, 33, 3, 4, 72, 50, dict(score="sigmoid")), (12, 2, 9, 3, 72, 50, {})])
def test_gated_experts_with_identities(T, E, ident, top, W, ff, kw, dtype):
    """Both forms of the experts; decisions are far apart and some hang on the correction."""
    from pocketllm_b200.models import mixer_layers as ml
    from pocketllm_b200.ops import mixer_ops as mo
    kw = {"score": "softmax", "renorm": True, "on_output": True, **kw}
    g = torch.Generator().manual_seed(T + E)
    r = lambda *s: torch.randn(*s, generator=g).to(BF16).float()
    n = E + ident
    x = r(T, W)
    gate, up, down = r(E, ff, W) * W ** -0.5, r(E, ff, W) * W ** -0.5, r(E, W, ff) * ff ** -0.5
    order = torch.stack([torch.randperm(n, generator=g) for _ in range(T)])
    corr = torch.zeros(n)
    corr[0] = 3.0                                                   # always chosen
    m = ml.RoutedExperts(r(n, W) * 0.02, list(up), list(down), mo.Router(E, top, identity=ident, **kw), dtype, "cuda", gate=list(gate), correction=corr)
    z = torch.zeros(T, m.router.N)
    z[:, :n].scatter_(1, order, torch.linspace(2.0, -2.0, n).repeat(T, 1) if n < 50 else torch.linspace(2.0, -20.0, n).repeat(T, 1))
    z[:, n:] = 50.0
    zc = z.cuda()
    m.router = lambda ctx, h, name, dt: zc
    ctx = ml.StepContext(T, *[None] * 6, ml.Workspace("cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"))
    h = torch.zeros(T, m.up.shape[2], device="cuda", dtype=dtype)
    h[:, :W] = x.to(dtype)
    got = torch.zeros(T, W, device="cuda")
    mo.sandwich_norm(got, eps=1e-5, plus_one=False, **m.forward(ctx, h))
    want = plain_experts(z[:, :n].double(), x.double(), gate.to(dtype).double(), up.to(dtype).double(), down.to(dtype).double(), top, corr.double(),
                         kw["renorm"], kw["on_output"], kw["score"])
    assert ((got.double().cpu() - want).norm() / want.norm()).item() < (1e-5 if dtype == F32 else 8e-3)
    assert int(ctx.status) == 0


# ---- every mechanism alone ----

ALONE = {
    "attention": config([attention()]),
    "attention_full": config([attention(window=None)]),
    "attention_window1": config([attention(window=1)]),
    "attention_window_huge": config([attention(window=100000)]),
    "attention_no_rot": config([attention(rot=0)]),
    "attention_all_rot": config([attention(dim=24, rot=24, factor=None, base=40.0)]),
    "attention_one": config([attention(heads=1, kv=1, dim=2, vdim=1, rot=2, window=5, scale=1.0)]),
    "attention_group": config([attention(heads=12, kv=1, dim=16, vdim=64, rot=16, window=65)]),      # two blocks of query vectors per key head
    "attention_128": config([attention(heads=2, kv=1, dim=128, vdim=128, rot=64, window=64, scale=0.09)]),
    "attention_values": config([attention(heads=2, kv=2, dim=60, rot=20, vdim=150, window=70)]),     # several value slices
    "attention_wide_keys": config([attention(heads=2, kv=1, dim=260, rot=16, vdim=20, window=33, scale=0.06)]),   # beyond the tensor-core form
    "attention_negative_scale": config([attention(scale=-0.2)]),
    "attention_steep": config([attention(window=None, scale=2.0)]),                                  # maxima that grow along the row
    "values_mixed": config([attention(v_mix=False), attention(), attention(v_mix=False, vdim=9), attention(factor=None, window=8), attention(heads=2)]),
    "parallel": config([parallel()]),
    "parallel_small_cap": config([parallel(cap=0.3)]),
    "parallel_large_cap": config([parallel(cap=500.0, left={"scale": 3.0})]),
    "parallel_window1": config([parallel(left={"window": 1})]),
    "parallel_full": config([parallel(left={"window": None, "rot": 18, "factor": 4.0})]),
    "parallel_no_rot": config([parallel(left={"rot": 0})]),
    "parallel_values": config([parallel(left={"heads": 2, "kv": 1, "dim": 30, "vdim": 150, "window": 70})]),
    "parallel_odd": config([parallel(left={"heads": 3, "kv": 3, "dim": 7, "vdim": 5, "rot": 6}, heads_=3, vdim=7, state=5, groups=3, parts=7, conv=2)]),
    "parallel_wide_keys": config([parallel(left={"heads": 2, "kv": 1, "dim": 260, "scale": 0.06})]),
    "parallel_negative": config([parallel(left={"scale": -0.3}, scales=(-0.8, 1.0))]),
    "space_one": config([parallel(heads_=1, vdim=1, state=1, groups=1, parts=1, conv=1)]),
    "space_taps1": config([parallel(conv=1)]),
    "space_taps2": config([parallel(conv=2, groups=6)]),
    "space_taps3": config([parallel(conv=3, groups=2)]),
    "space_taps7": config([parallel(conv=7, groups=1, parts=1)]),
    "space_taps12": config([parallel(conv=12, parts=60)]),
    "space_wide": config([parallel(heads_=4, vdim=70, state=130, groups=2, parts=8)]),
    "space_64": config([parallel(heads_=4, vdim=64, state=64, groups=4, parts=2)]),
    "space_big": config([parallel(heads_=2, vdim=128, state=256, groups=1, parts=1)], width=64),
    "space_long_parts": config([parallel(heads_=36, vdim=64, state=16, groups=4, parts=1)], width=64),
    "experts": config([attention(moe(experts=6, identity=3, top=4, ff=130))], width=65),
    "experts_one": config([attention(moe(experts=1, identity=0, top=1, ff=20))]),
    "experts_identity_only_left": config([attention(moe(experts=1, identity=1, top=1, ff=20))]),
    "experts_all": config([parallel(moe(experts=3, identity=2, top=5, ff=70))]),
    "multiplier_one": config([parallel(moe()), attention()], mult=1.0),
    "multiplier_negative": config([parallel(), attention(moe())], mult=-0.7),
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


@pytest.mark.parametrize("steps", ["fast", "slow"])
def test_decays_at_both_ends(steps):
    """Decays that forget within a token, and decays under which the first token is still in the state, and in the logits, after
    hundreds."""
    cfg = config([parallel(left={"window": 3}, scales=(0.2, 1.5))])
    t = tensors(cfg, 4)
    fast = steps == "fast"
    t["l0.mix.right.A_log"] = torch.full((6,), 4.0 if fast else -7.0).to(BF16)
    t["l0.mix.right.dt_bias"] = torch.full((6,), 3.0 if fast else -3.0).to(BF16)
    seq = tokens(400, cfg["vocab"], 8)
    want = zr.PlainModel(cfg, t).logits(seq)
    if not fast:
        other = zr.PlainModel(cfg, t).logits([(seq[0] + 1) % 83] + seq[1:])
        assert ((want - other).pow(2).mean(-1).sqrt() / want.std())[390] > 1e-3
    rt = runtime(cfg, t)
    check(feed(rt, "a", seq, [400]), want)
    check(feed(rt, "a", seq, [200, 1, 130, 1]), want)


@pytest.mark.parametrize("taps", [2, 4, 5])
def test_convolution_at_portion_edges(taps):
    """The line of the convolution over portions shorter and longer than it, in a slot that another request has left."""
    cfg = config([parallel(conv=taps, scales=(0.1, 1.5))])
    t = tensors(cfg, 6)
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
    """The residual stream behind every layer, in prompts and single tokens."""
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
            rt.step([StepEntry("a", seq[a:b])])
        n = len(FULL["layers"])
        got = [torch.cat(rt.launch_layers[i::n]).double().cpu() for i in range(n)]
        for i in range(n):
            assert ((got[i] - want[i]).norm() / want[i].norm()).item() < (2e-6 if dtype == F32 else 2e-2)


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
@pytest.mark.parametrize("kind,window", [("attention", 29), ("attention", 64), ("attention", None), ("parallel", 37), ("parallel", 65)])
def test_keys_at_window_and_page_edges(kind, window, dtype):
    """One key stands out: seen up to the last position of its window and not one later, at page borders, at the start of the
    sequence and far back; in prompts, short portions and single tokens."""
    if kind == "attention":
        cfg = config([attention(window=window), attention(heads=1, kv=2 // 2, dim=4, vdim=13, rot=2, v_mix=False)])
    else:
        cfg = config([parallel(left={"window": window}, cap=30.0, scales=(1.0, 0.05))])
    t = beacon_tensors(cfg)
    m = zr.PlainModel(cfg, t)
    rt = runtime(cfg, t, dtype)
    for place in (0, 20, 28, 63, 64, 75):
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


@pytest.mark.parametrize("kind", ["attention", "parallel"])
def test_split_context_decode(kind):
    """Context long enough for several splits of the row kernel, with a far key that stands out."""
    far = {"window": None, "heads": 3, "kv": 1}
    cfg = config([attention(**far) if kind == "attention" else parallel(left=far, cap=30.0, scales=(1.0, 0.05))])
    t = beacon_tensors(cfg)
    seq = tokens(600, cfg["vocab"], 77, low=1)
    seq[37] = BEACON
    want = zr.PlainModel(cfg, t).logits(seq)
    for dtype in (F32, BF16):
        rt = runtime(cfg, t, dtype, pages=24)
        m = rt.model.layers[0].mixer
        assert getattr(m, "left", m).nsplit > 4
        check(feed(rt, "a", seq, [590, 1]), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """280 single tokens after a short prompt, through graphs, over several pages and windows."""
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
    zm.save_checkpoint(tmp_path / "m", zm.ZemozenConfig.from_dict(FULL), t)
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
