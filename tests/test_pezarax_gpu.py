"""Pezarax on the GPU against the plain oracle (float64, token by token): every mechanism alone, prompts, portions, mixed
batches, reused pages and slots, chunk edges, long decoding, unusual sizes, generation through the scheduler, the CLI; and the
variants that the new kernels offer to other designs."""
import json
import subprocess
import sys
from pathlib import Path

import pezarax_reference as pr
import pytest
import torch
from mixer_checks import BF16, F32, check, feed, make_runtime, margin_prefix, traffic
from mixer_reference import rms, rotate_half
from pezarax_cases import BEACON, FULL, attention, beacon_tensors, clear_routes, config, moe, retention, tensors, tokens

from pocketllm_b200.models import pezarax as pz
from pocketllm_b200.server.engine import SamplingParams

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def runtime(cfg, t, dtype=F32, **kw):
    return make_runtime(pz, pz.PezaraxConfig, cfg, t, dtype, **kw)


_memo: dict = {}


def oracle(cfg, t, seq, key):
    k = (key, len(seq))
    if k not in _memo:
        _memo[k] = pr.PlainModel(cfg, t).logits(seq)
    return _memo[k]


# ---- kernels ----

@pytest.mark.parametrize("W", [24, 300, 2048])
def test_residual_steps_without_post_norm(W):
    """Plain addition of a sublayer's output, of the sum of a token's expert rows, of the scaled embedding row."""
    from pocketllm_b200.ops import mixer_ops as mo
    T, V, eps, sc = 5, 9, 1e-3, 3.25
    x, y, wn = torch.randn(T, W, device="cuda"), torch.randn(3 * T, W + 4, device="cuda"), torch.randn(W, device="cuda")
    emb = torch.randn(V, W, device="cuda").to(BF16)
    toks = torch.tensor([0, 3, V - 1, 5, 5], dtype=torch.int32, device="cuda")
    place = torch.randperm(3 * T, device="cuda").to(torch.int32).view(T, 3)
    e = emb[toks.long()].float() * sc
    kw = dict(eps=eps, plus_one=False)
    for step, want in ((dict(y=y[:T]), x + y[:T, :W]), (dict(y=y, y_rows=place), x + y[place.long(), :W].sum(1)),
                       (dict(tokens=toks, embed=emb, embed_scale=sc), e),
                       (dict(y=y[:T], tokens=toks, embed=emb, embed_scale=sc, embed_add=True), x + y[:T, :W] + e)):
        a, out = x.clone(), torch.full((T, W + 8), 7.0, device="cuda")
        mo.sandwich_norm(a, w_pre=wn, out=out, **step, **kw)
        assert torch.allclose(a, want, atol=1e-5)
        assert torch.allclose(out[:, :W], rms(want, eps) * wn, atol=1e-4, rtol=1e-4) and (out[:, W:] == 0).all()


def plain_experts(z, x, up, down, top, score="sigmoid", renorm=False, scale=1.0, on_output=False):
    s = torch.sigmoid(z) if score == "sigmoid" else torch.softmax(z, -1)
    w, ids = s.topk(top, -1)
    if renorm:
        w = w / w.sum(-1, keepdim=True)
    w = w * scale
    y = torch.zeros(x.shape[0], down.shape[1], dtype=x.dtype, device=x.device)
    for t in range(x.shape[0]):
        for j in range(top):
            e, f = ids[t, j], w[t, j]
            h = torch.relu(up[e] @ (x[t] if on_output else f * x[t])) ** 2
            y[t] += down[e] @ h * (f if on_output else 1)
    return y


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,E,top,W,ff,kw", [
    (1, 5, 2, 72, 36, {}), (8, 3, 1, 130, 200, {}), (37, 7, 3, 72, 36, {}), (150, 6, 6, 264, 130, {}), (300, 100, 2, 64, 128, {}), (3, 512, 32, 64, 20, {}),
    (20, 1, 1, 48, 40, {}), (40, 9, 2, 72, 50, dict(on_output=True)), (4, 9, 2, 72, 50, dict(on_output=True, renorm=True)),
    (30, 33, 4, 72, 50, dict(score="softmax", renorm=True, scale=1.7)), (5, 33, 4, 72, 50, dict(score="softmax", scale=2.0))])
def test_routed_experts(T, E, top, W, ff, kw, dtype):
    """Both forms of the experts, with the router's variants; decisions are far apart."""
    from pocketllm_b200.models import mixer_layers as ml
    from pocketllm_b200.ops import mixer_ops as mo
    g = torch.Generator().manual_seed(T + E)
    r = lambda *s: torch.randn(*s, generator=g).to(BF16).float()
    x = r(T, W)
    router, up, down = r(E, W) * 0.02, r(E, ff, W) * W ** -0.5, r(E, W, ff) * ff ** -0.5
    order = torch.stack([torch.randperm(E, generator=g) for _ in range(T)])
    m = ml.RoutedExperts(router, list(up), list(down), mo.Router(E, top, **kw), dtype, "cuda")
    # logits with gaps, in place of the router's product
    z = torch.zeros(T, m.router.N)
    z[:, :E].scatter_(1, order, torch.linspace(2.0, -2.0, E).repeat(T, 1) if E < 50 else torch.linspace(2.0, -20.0, E).repeat(T, 1))
    z[:, E:] = 50.0                                                   # padding columns are nobody's experts
    zc = z.cuda()
    m.router = lambda ctx, h, name, dt: zc
    ctx = ml.StepContext(T, *[None] * 6, ml.Workspace("cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"))
    h = torch.zeros(T, m.up.shape[2], device="cuda", dtype=dtype)
    h[:, :W] = x.to(dtype)
    out = m.forward(ctx, h)
    y, rows = out["y"], out.get("y_rows")
    got = (y if rows is None else y[rows.long()].sum(1))[:, :W].double().cpu()
    want = plain_experts(z[:, :E].double(), x.double(), up.to(dtype).double(), down.to(dtype).double(), top, **kw)
    assert ((got - want).norm() / want.norm()).item() < (1e-5 if dtype == F32 else 8e-3)
    assert int(ctx.status) == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,V,rot,window", [(4, 2, 24, 40, 8, None), (3, 1, 64, 64, 64, 33), (8, 8, 130, 200, 0, 70), (12, 1, 16, 8, 16, 1), (2, 2, 300, 20, 30, 50)])
def test_plain_grouped_attention(H, G, D, V, rot, window, dtype):
    """The attention layer without a second map: full or in a window, as another design would use it."""
    from pocketllm_b200.models import mixer_layers as ml
    from pocketllm_b200.runtime.mixer_runtime import MixerRuntime
    W, vocab = 56, 61
    g = torch.Generator().manual_seed(D)
    r = lambda *s: torch.randn(*s, generator=g).to(BF16)
    b = lambda *s: (torch.randn(*s, generator=g) * s[1] ** -0.5).to(BF16)
    w = {"q": b(H * D, W) * 2, "k": b(G * D, W) * 2, "v": b(G * V, W), "o": b(W, H * V)}
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": D ** -0.5}
    if rot:
        m["rot"] = {"base": 900.0, "dims": rot}
    if window:
        m["mask"] = {"size": window}
    embed, head, n1 = r(vocab, W), b(vocab, W), torch.ones(W)
    mixer = ml.GroupedAttentionMixer(w, m, 1e-5, dtype, "cuda", 6, 384)
    model = ml.MixerModel(vocab, W, 1e-5, dtype, embed.cuda(), [ml.MixerLayer(mixer, n1.cuda())], n1.cuda(), ml.FusedLinear([("head", head)], dtype, "cuda"),
                          plus_one=False)
    rt = MixerRuntime(model, max_requests=2, pages=6)
    seq = tokens(160, vocab, 2)
    x = embed.double()[seq]
    h = rms(x, 1e-5)
    turn = lambda a: torch.stack([rotate_half(a[p], p, m["rot"]) for p in range(160)]) if rot else a
    q, k, v = turn((h @ w["q"].double().t()).view(160, H, D)), turn((h @ w["k"].double().t()).view(160, G, D)), (h @ w["v"].double().t()).view(160, G, V)
    i = torch.arange(160)
    see = (i[None] <= i[:, None]) & (i[None] > i[:, None] - (window or 1000))
    o = []
    for a in range(H):
        s = (q[:, a] @ k[:, a // (H // G)].t() * D ** -0.5).masked_fill(~see, -torch.inf)
        o.append(torch.softmax(s, -1) @ v[:, a // (H // G)])
    x = x + torch.cat(o, -1) @ w["o"].double().t()
    want = rms(x, 1e-5) @ head.double().t()
    for cuts in ([160], [1], [70, 1, 2, 9, 1, 64, 3]):
        check(feed(rt, "a", seq, cuts), want, dtype)


# ---- every mechanism alone ----

ALONE = {
    "retention": config([retention()]),
    "retention_wide": config([retention(heads=2, dim=70, vdim=33, rot=38)]),
    "retention_plain": config([retention(rot=0, heads=1, dim=33, vdim=65, decay=(0.98,))]),
    "retention_one": config([retention(heads=1, dim=1, vdim=1, rot=0)]),
    "retention_pair": config([retention(heads=2, dim=2, vdim=3, rot=2, base=10.0)]),
    "retention_big": config([retention(heads=1, dim=260, vdim=140, rot=260)], width=64),
    "retention_decays": config([retention(heads=5, decay=(0.0, 1.0, 0.01, 0.999999, 0.5))]),
    "attention": config([attention()]),
    "attention_full": config([attention(chunk=None)]),
    "attention_chunk1": config([attention(chunk=1)]),
    "attention_chunk_huge": config([attention(chunk=100000)]),
    "attention_one": config([attention(heads=1, kv=1, dim=2, vdim=1, rot=2, chunk=5, scale=1.0)]),
    "attention_group": config([attention(heads=12, kv=1, dim=16, vdim=64, rot=16, chunk=65)]),            # two blocks of query vectors per key head
    "attention_128": config([attention(heads=2, kv=1, dim=128, vdim=128, rot=64, chunk=64, scale=0.09)]),  # widest form with both maps in a block
    "attention_values": config([attention(heads=2, kv=2, dim=60, rot=20, vdim=150, chunk=70)]),            # several value slices
    "attention_keys": config([attention(heads=2, kv=1, dim=150, rot=16, vdim=20, chunk=33, scale=0.08)]),  # one map per block
    "attention_wide_keys": config([attention(heads=2, kv=1, dim=260, rot=16, vdim=20, chunk=33, scale=0.06)]),   # beyond the tensor-core form
    "attention_negative_scale": config([attention(scale=-0.2)]),
    "attention_steep": config([attention(chunk=None, scale=4.0)]),                                         # maxima that grow along the row
    "attention_no_rot": config([attention(rot=0, diff=0.0)]),
    "experts": config([retention(mlp=moe(experts=6, top=3, ff=130))], width=65),
    "experts_one": config([retention(mlp=moe(experts=1, top=1, ff=20))]),
    "experts_all": config([attention(mlp=moe(experts=3, top=3, ff=70))]),
    "loop": config([retention(), attention(), retention(heads=1)], loop=(0, 2, 3)),
    "loop_one": config([retention(), attention(chunk=16)], loop=(1, 2, 2)),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(ALONE))
def test_mechanism_alone(name, dtype):
    cfg = ALONE[name]
    t = clear_routes(cfg, tensors(cfg, 3))
    seq = tokens(140, cfg["vocab"], 1)
    want = oracle(cfg, t, seq, "alone " + name)
    rt = runtime(cfg, t, dtype)
    check(feed(rt, "p", seq, [140]), want, dtype)
    check(feed(rt, "d", seq, [1]), want, dtype)
    check(feed(rt, "m", seq, [70, 1, 2, 9, 1, 64, 3]), want, dtype)


def test_hundreds_of_decayed_tokens():
    """Slow decays over many chunks of the scan: what the first tokens left is still in the state, and in the logits."""
    cfg = config([retention(heads=2, decay=(0.9999, 0.99))])
    t = tensors(cfg, 4)
    seq = tokens(500, cfg["vocab"], 8)
    want = pr.PlainModel(cfg, t).logits(seq)
    other = pr.PlainModel(cfg, t).logits([(seq[0] + 1) % 83] + seq[1:])
    assert ((want - other).pow(2).mean(-1).sqrt() / want.std())[490] > 2e-3
    rt = runtime(cfg, t)
    check(feed(rt, "a", seq, [500]), want)
    check(feed(rt, "a", seq, [300, 1, 130, 1]), want)


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
    want = pr.PlainModel(FULL, t).logits(seq)
    rt = runtime(FULL, t)
    check(feed(rt, "a", seq, [120]), want)
    check(feed(rt, "a", seq, [50, 1, 8, 40]), want)


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
@pytest.mark.parametrize("chunk,chosen", [(29, 0), (64, 1), (65, 0), (None, 1)])
def test_keys_at_chunk_and_page_edges(chunk, chosen, dtype):
    """One key stands out in one of the maps: seen up to the last position of its chunk and not one later, at page borders, at
    the start of the sequence and far back; in prompts, short portions and single tokens."""
    cfg = config([attention(chunk=chunk), retention(heads=1, dim=4, vdim=6, rot=2)])
    t = beacon_tensors(cfg, chosen_map=chosen)
    m = pr.PlainModel(cfg, t)
    rt = runtime(cfg, t, dtype)
    for place in (0, 20, 28, 63, 64, 87):
        seq = tokens(140, cfg["vocab"], 30 + place, low=1)
        seq[place] = BEACON
        want = m.logits(seq)
        check(feed(rt, "p", seq, [140]), want, dtype)
        check(feed(rt, "d", seq, [max(1, place - 3), 1]), want, dtype)
        check(feed(rt, "s", seq, [place + 7, 2, 2, 2, 8]), want, dtype)
        check(feed(rt, "c", seq, [place + 11, 33]), want, dtype)


def test_first_tokens():
    t = full_tensors(5)
    for n in (1, 2, 3):
        seq = tokens(n, FULL["vocab"], 90 + n)
        want = pr.PlainModel(FULL, t).logits(seq)
        for dtype in (F32, BF16):
            rt = runtime(FULL, t, dtype)
            check(feed(rt, "a", seq, [n]), want, dtype)
            check(feed(rt, "a", seq, [1]), want, dtype)


def test_split_context_decode():
    """Context long enough for several splits of the row kernel, with a far key that stands out."""
    cfg = config([attention(chunk=None, heads=3, kv=1)])
    t = beacon_tensors(cfg)
    seq = tokens(600, cfg["vocab"], 77, low=1)
    seq[37] = BEACON
    want = pr.PlainModel(cfg, t).logits(seq)
    for dtype in (F32, BF16):
        rt = runtime(cfg, t, dtype, pages=24)
        assert rt.model.layers[0].mixer.nsplit > 4
        check(feed(rt, "a", seq, [590, 1]), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """280 single tokens after a short prompt, through graphs, over several pages and chunks."""
    t = full_tensors(11)
    seq = tokens(300, FULL["vocab"], 6)
    want = oracle(FULL, t, seq, "long")
    check(feed(runtime(FULL, t, dtype), "a", seq, [20, 1]), want, dtype)


def test_greedy_generation_through_the_scheduler():
    from pocketllm_b200.runtime.batching import BatchEngine
    from pocketllm_b200.server.backends import MixerBackend
    from pocketllm_b200.server.engine import ServingEngine
    t = full_tensors(12)
    m = pr.PlainModel(FULL, t)
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
    pz.save_checkpoint(tmp_path / "m", pz.PezaraxConfig.from_dict(FULL), t)
    ids = [ord(c) % 101 for c in "Qy7 =b"]
    r = subprocess.run([sys.executable, "-m", "pocketllm_b200.cli.generate", "--ckpt-path", str(tmp_path / "m"), "--tokenizer-path", "chars", "--prompt",
                        "".join(chr(i) for i in ids), "--max-new-tokens", "6", "--max-context", "256", "--dtype", "float32"],
                       cwd=ROOT, capture_output=True, timeout=280)
    assert r.returncode == 0, r.stderr.decode()
    want = pr.PlainModel(FULL, t).generate(ids, 6)
    assert r.stdout.decode() == "".join(chr(i) for i in want) + "\n"
    seq = tokens(70, 101, 3)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seq[:40], "want": [39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": seq[40:41], "want": []}, {"id": "b", "tokens": seq[:30], "want": [0, 29]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": seq[30:31], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": seq, "want": [69]}], "end": ["c"]}]
    ref = pr.PlainModel(FULL, t).logits(seq)
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
