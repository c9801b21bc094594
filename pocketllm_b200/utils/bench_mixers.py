"""Throughput of mixer decoders (Gidisun) at sizes that resemble a real model's layers, beside the closest existing model at
equal size (the Qwen hybrid: DeltaNet + GQA, same width, feed-forward, depth and vocabulary), and the time of each new
kernel beside the like kernel of the existing families.

    python -m pocketllm_b200.utils.bench_mixers --kernels
    python bench.py --model gidisun [--size 2k|4k]

Random weights; every weight set is larger than L2. Device times by CUDA events.
"""
from __future__ import annotations

import argparse
import json

import torch

from ..models import gidisun as gd

VOCAB = 32000
#            width  ff     mLSTM (heads, dim, vdim)  GLA              latent (heads, dim, rot, vdim, rank, window)
SIZES = {"2k": (2048, 6144, (8, 128, 256), (16, 128, 128), (16, 128, 64, 128, 512, 1024)),
         "4k": (4096, 14336, (8, 256, 512), (16, 128, 256), (32, 128, 64, 128, 512, 1024))}
PATTERN = ("mlstm", "latent_attention", "gla", "gla", "mlstm", "latent_attention", "gla", "mlstm")


def config(size: str) -> gd.GidisunConfig:
    W, ff, m, g, a = SIZES[size]
    mix = {"mlstm": {"heads": m[0], "dim": m[1], "vdim": m[2], "gate_cap": 12.0},
           "gla": {"heads": g[0], "dim": g[1], "vdim": g[2], "tau": 14.0},
           "latent_attention": {"heads": a[0], "dim": a[1], "rot_dim": a[2], "vdim": a[3], "kv_rank": a[4], "scale": (a[1] + a[2]) ** -0.5,
                                "mask": {"size": a[5]}, "rot": {"base": 5e5, "dims": a[2],
                                                                "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}}
    return gd.GidisunConfig.from_dict({"architecture": gd.ARCH, "vocab": VOCAB, "width": W, "norm": {"eps": 1e-5},
                                       "layers": [{"type": t, "mixer": mix[t], "mlp": {"kind": "dense", "ff": ff}} for t in PATTERN]})


def build(size: str, batch: int, context: int):
    from ..runtime.mixer_runtime import MixerRuntime
    c = config(size)
    t = {n: v.cpu() for n, v in gd.random_tensors(c, 0, device="cuda").items()}
    pages = batch * (-(-context // 64))
    streamed = sum(v.numel() for n, v in t.items() if n != "embed") * 2
    return MixerRuntime(gd.build_model(c, t, slots=batch, pages=pages), max_requests=batch, pages=pages), streamed


def closest_model(size: str, prompt: int, decode: int, reps: int) -> dict:
    """Single-request prefill and decode of the Qwen hybrid at the same width, feed-forward, depth and vocabulary (FP8 weights:
    half the bytes per weight)."""
    from ..models import qwen_hybrid as qh
    W, ff = SIZES[size][:2]
    cfg = qh.QwenHybridConfig(vocab_size=VOCAB, hidden_size=W, intermediate_size=ff, num_hidden_layers=len(PATTERN), num_attention_heads=W // 128,
                              num_key_value_heads=W // 512, linear_num_key_heads=W // 256, linear_num_value_heads=W // 128,
                              max_position_embeddings=8192)
    eng = qh.QwenEngine(cfg, max_context=prompt + decode + 16, prefill_chunk=min(prompt, 2048)).init_random(0, 0.02)
    g = torch.Generator().manual_seed(0)
    p = torch.randint(0, VOCAB, (prompt,), generator=g).tolist()
    pre = dec = 0.0
    for i in range(3 + reps):
        eng.reset()
        eng.prefill(p)
        eng.decode(decode)
        t = eng.timings()
        if i >= 3:
            pre, dec = pre + t["prefill_ms"], dec + t["decode_ms"]
    out = {"model": "Qwen hybrid (DeltaNet + GQA, FP8 weights)", "prefill_tok_s": round(reps * prompt / pre * 1e3, 1),
           "decode_tok_s": round(reps * decode / dec * 1e3, 1), "weight_gb": round(eng.weight_bytes / 1e9, 2)}
    eng.close()
    return out


def timed(fn, reps: int = 20, warmup: int = 5) -> float:
    """Mean microseconds of one call, captured as a graph of `reps` calls: host overhead stays off the timeline."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for _ in range(reps):
            fn()
    g.replay()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    g.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps * 1e3


def _roof(us: float, flops: float = 0.0, nbytes: float = 0.0) -> dict:
    """Fractions of the measured copy bandwidth, of the bf16 burst rate and of the fp32 lanes (148 x 128 fma at 1.965 GHz)."""
    from .bench_kernels import peaks
    hbm, tf, src = peaks()
    out = {"us": round(us, 2)}
    if nbytes:
        out.update(gbs=round(nbytes / us / 1e3, 1), frac_copy=round(nbytes / us / 1e3 / hbm, 3))
    if flops:
        out.update(tflops=round(flops / us / 1e6, 2), frac_fp32_simt=round(flops / us / 1e6 / 74.4, 3), frac_bf16=round(flops / us / 1e6 / tf, 4))
    return out


class _Batch:
    """A step context over made-up positions: `T` rows of one request at `start`, as one long portion or as single rows."""

    def __init__(self, T: int, start: int, context: int, windows=(0,), singles: bool = False):
        from ..models.mixer_layers import StepContext, Workspace
        from ..runtime.mixer_runtime import plan_portions
        p = plan_portions([1] * T, [start] * T, list(range(T)), windows) if singles else plan_portions([T], [start], [0], windows)
        dev = lambda a: torch.as_tensor(a, dtype=torch.int32).cuda().contiguous()
        slots, pages = (T if singles else 1), -(-context // 64)
        table = dev(range(slots * pages)).view(slots, pages)
        self.pages, self.slots = slots * pages, slots
        self.ctx = StepContext(T, dev([0] * T), dev(p["pos"]), dev(p["slot"]), dev(p["last"]), table, Workspace("cuda"),
                               torch.zeros(1, dtype=torch.int32, device="cuda"), short=dev(p["short"]), n_short=len(p["short"]), rows=dev(p["rows"]),
                               n_rows=len(p["rows"]), all_rows=dev(range(T)), long=dev(p["long"]), n_long=len(p["long"]), chunks=dev(p["chunks"]),
                               chunk0=dev(p["chunk0"]), n_chunks=len(p["chunks"]), tiles=dev(p["tiles"]), n_tiles=len(p["tiles"]),
                               gather={w: (dev(p["gather"][w]), p["total"][w], p["longest"][w]) for w in windows})


def _state(kind: str, dims, T: int, singles: bool):
    """The recurrence of one layer (without its projections): (call, flops, bytes)."""
    from ..models import mixer_layers as ml
    from ..ops import mixer_ops as mo
    H, D, V = dims
    W = 1024
    b = _Batch(T, 4096, 64, singles=singles)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    w = {"q": r(H * D, W), "k": r(H * D, W), "v": r(H * V, W), "g": r(H * V, W), "o": r(W, H * V)}
    if kind == "mlstm":
        w.update({"i": r(H, W), "f": r(H, W), "i.b": torch.zeros(H), "f.b": torch.full((H,), 3.0), "norm": torch.ones(H * V)})
        m = ml.MLSTMMixer(w, {"heads": H, "dim": D, "vdim": V, "gate_cap": 12.0}, 1e-5, torch.bfloat16, "cuda", b.slots)
    else:
        w.update({"a1": r(16, W), "a2": r(H * D, 16), "a2.b": torch.full((H * D,), 2.0), "norm": torch.ones(V)})
        m = ml.GLAMixer(w, {"heads": H, "dim": D, "vdim": V, "tau": 14.0}, 1e-5, torch.bfloat16, "cuda", b.slots)
    ctx, ws = b.ctx, b.ctx.ws
    p = m.proj(ctx, torch.randn(T, m.proj.K, device="cuda").to(torch.bfloat16), "proj", torch.float32)
    o, nq, mm = ws.flat("o", T * H * V, torch.float32), ws.flat("nq", T * H, torch.float32), ws.flat("m", T * H, torch.float32)
    d = mo.StateMixer(proj=p.data_ptr(), ld=p.stride(0), o=o.data_ptr(), nq=nq.data_ptr(), m=mm.data_ptr(), **m.desc)
    mix = ws.rows("mix", T, m.out.K, torch.bfloat16)
    scratch = ws.flat("ws", mo.state_chunk_workspace(d, max(ctx.n_chunks, 1)), torch.float32)

    def call():
        if singles:
            mo.state_rows(d, ctx.short, ctx.n_short)
        else:
            mo.state_chunks(d, ctx.long, 1, ctx.chunks, ctx.chunk0, ctx.n_chunks, scratch)
        mo.state_out(d, m.norm, m.per_head_norm, 1e-5, ctx.last_slot, T, mix)
    call.keep = (m, b, p)
    flops = 2.0 * T * H * (2 * D * V + 64 * D + 64 * V)
    return call, flops, T * H * D * V * 8.0 if singles else 0.0


def _latent(dims, T: int, start: int, singles: bool):
    """The attention of one latent layer after its input projection, without the output projection; returns
    {kernel: (call, flops, bytes)}."""
    from ..models import mixer_layers as ml
    from ..ops import mixer_ops as mo
    H, D, R, V, K, window = dims
    W = 1024
    b = _Batch(T, start, start + T, windows=(window,), singles=singles)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    m = ml.LatentAttentionMixer({"q": r(H * (D + R), W), "dkv": r(K + R, W), "dkv.norm": torch.ones(K), "uk": r(H * D, K), "uv": r(H * V, K),
                                 "sink": torch.zeros(H), "o": r(W, H * V)},
                                {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": K, "scale": (D + R) ** -0.5,
                                 "mask": {"size": window} if window else None, "rot": {"base": 1e4, "dims": R}}, 1e-5, torch.bfloat16, "cuda",
                                b.pages, start + T)
    m.cache.normal_()
    ctx, ws = b.ctx, b.ctx.ws
    p = m.proj(ctx, torch.randn(T, m.proj.K, device="cuda").to(torch.bfloat16), "proj", torch.float32)
    qw = m.qk_panels * 64
    mix = ws.rows("mix", T, m.out.K, torch.bfloat16)
    span = sum(min(start + i + 1, window or 1 << 30) for i in range(T)) if not singles else T * min(start + 1, window or 1 << 30)
    keep = (m, b, p)
    if singles:
        qx = ws.flat("qx", T * H * m.row, torch.float32)
        po, pm = ws.flat("po", T * m.nsplit * H * K, torch.float32), ws.flat("pm", T * m.nsplit * H * 2, torch.float32)
        return {"prep": (lambda k=keep: mo.latent_prep(p, 0, m.proj.at["dkv"], H, D, R, K, m.c_norm, 1e-5, m.freq, m.mag, ctx.pos, ctx.slot, m.cache,
                                                       ctx.table, qx, None, qw), 0, 0),
                "absorb": (lambda: mo.latent_absorb(p, 0, H, D, R, K, m.uk, ctx.rows, T, qx, m.row), 2.0 * T * H * D * K, H * D * K * 2.0),
                "rows": (lambda: mo.latent_rows(qx, ctx.rows, T, ctx.pos, ctx.slot, m.cache, ctx.table, H, K, m.window, m.scale, m.nsplit, po, pm),
                         2.0 * span * H * (m.row + K), span * m.row * 2.0),
                "merge + values": (lambda: mo.latent_out(po, pm, m.nsplit, H, K, V, m.sink, ctx.rows, T, m.uv, mix), 2.0 * T * H * V * K, H * V * K * 2.0)}
    qf = ws.flat("qf", T * H * qw, torch.bfloat16)
    gather, total, longest = ctx.gather[m.window]
    c, kv = ws.rows("c", total, m.row, torch.bfloat16), ws.rows("kv", total, m.kv_w.shape[0], torch.bfloat16)
    return {"prep": (lambda k=keep: mo.latent_prep(p, 0, m.proj.at["dkv"], H, D, R, K, m.c_norm, 1e-5, m.freq, m.mag, ctx.pos, ctx.slot, m.cache,
                                                   ctx.table, None, qf, qw), 0, T * (p.shape[1] * 4.0 + m.row * 2 + H * qw * 2)),
            "gather": (lambda: mo.latent_gather(m.cache, ctx.table, ctx.long, gather, 1, longest, c), 0, total * m.row * 4.0),
            "expand": (lambda: mo.linear(c, m.kv_w, kv, ctx.status), 2.0 * total * m.row * kv.shape[1], 0),
            "attention": (lambda: mo.latent_prefill(qf, T, kv, total, ctx.tiles, ctx.n_tiles, ctx.long, gather, H, m.qk_panels, m.v_panels, V, m.window,
                                                    m.scale, m.sink, mix, ctx.status), 2.0 * span * H * (D + R + V), 0)}


def kernels() -> None:
    from .. import ops
    from ..ops import mixer_ops as mo
    from . import bench_kernels as bk
    show = lambda name, d, **kw: print(json.dumps({"kernel": name, **kw, **d}), flush=True)
    # recurrent layers: equal state (16 x 128 x 256 = 32 x 128 x 128)
    for T in (512, 2048):
        for kind, dims in (("gla", (16, 128, 256)), ("mlstm", (8, 256, 512))):
            f, fl, _ = _state(kind, dims, T, False)
            show(f"{kind} chunk form + head norm", _roof(timed(f), fl), T=T, dims=dims)
        r = bk.bench_deltanet(T, 16, 32, 20)
        show("like kernel: chunked DeltaNet", _roof(r["us"], 2.0 * T * 32 * (3 * 128 * 128 + 2.5 * 64 * 128 + 64 * 64 * 1.0)), T=T)
    for B in (1, 8):
        for kind, dims in (("gla", (16, 128, 256)), ("mlstm", (8, 256, 512))):
            f, _, nb = _state(kind, dims, B, True)
            show(f"{kind} rows form + head norm", _roof(timed(f), 0, nb), B=B, dims=dims)
    ld, C = (2 * 16 + 2 * 32) * 128 + 64, (2 * 16 + 32) * 128
    proj = torch.randn(1, ld, device="cuda").to(torch.bfloat16)
    z = lambda *s: torch.zeros(*s, device="cuda")
    st, cs, cw = z(32, 128, 128), z(C, 3), z(C, 4)
    show("like kernel: DeltaNet step", _roof(timed(lambda: ops.deltanet_seq(proj, 16, 32, cw, cs, z(32), z(32), z(128), 1e-6, st)), 0, 32 * 128 * 128 * 8.0), B=1)
    # attention of a long portion
    for dims, start in (((32, 128, 64, 128, 512, 0), 8192 - 512), ((32, 128, 64, 128, 512, 1024), 8192 - 512)):
        for k, (f, fl, nb) in _latent(dims, 512, start, False).items():
            show("latent prefill: " + k, _roof(timed(f), fl, nb), T=512, context=8192, window=dims[-1])
    show("like kernel: GQA prefill", bk.bench_attention(512, 8192, 32, 8, 20))
    # attention of single rows
    for B, win in ((1, 1024), (8, 1024), (64, 640)):
        for k, (f, fl, nb) in _latent((32, 128, 64, 128, 512, win), B, 1500, True).items():
            show("latent rows: " + k, _roof(timed(f), fl, nb), B=B, window=win)
    for M in (1, 8, 64):
        for r in bk.bench_dsv4_select_attend(M, 32768, 20):
            if "sparse_attn" in r["op"]:
                show("like kernel: sparse attention over 640 latent rows", r)
    # few-row linears and norms
    for M in (1, 4, 8):
        for N, K, sw in ((28672, 4096, True), (4096, 14336, False), (12416, 4096, False)):
            ws = [torch.randn(N, K, device="cuda").to(torch.bfloat16) for _ in range(max(2, -(-(300 << 20) // (N * K * 2))))]
            x = torch.randn(M, K, device="cuda").to(torch.bfloat16)
            y = torch.empty(M, N // 2 if sw else N, device="cuda", dtype=torch.bfloat16 if sw else torch.float32)
            s = torch.zeros(1, dtype=torch.int32, device="cuda")
            us = timed(lambda: [mo.linear(x, w, y, s, swiglu=sw) for w in ws], reps=8) / len(ws)
            show("few-row linear", _roof(us, 0, N * K * 2.0), M=M, N=N, K=K, swiglu=sw)
            if not sw:
                us = timed(lambda: [ops.matvec(x, None, None, w, epi=2) for w in ws], reps=8) / len(ws)
                show("like kernel: matvec on bf16 rows", _roof(us, 0, N * K * 2.0), M=M, N=N, K=K)
    for T in (1, 2048):
        x, y, w = torch.randn(T, 4096, device="cuda"), torch.randn(T, 4096, device="cuda"), torch.randn(4096, device="cuda")
        o = torch.empty(T, 4096, device="cuda", dtype=torch.bfloat16)
        show("sandwich norm", _roof(timed(lambda: mo.sandwich_norm(x, y=y, w_post=w, w_pre=w, out=o, eps=1e-5)), 0, T * 4096 * 14.0), T=T)
        xb = x.to(torch.bfloat16)
        show("like kernel: RMSNorm with residual add", _roof(timed(lambda: ops.rmsnorm(xb, w, parts=y[None], hidden_out=o)), 0, T * 4096 * 10.0), T=T)


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--size", default="2k", choices=sorted(SIZES))
    args = ap.parse_args()
    if args.kernels:
        kernels()
    else:
        print(json.dumps(closest_model(args.size, 512, 64, 3)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
