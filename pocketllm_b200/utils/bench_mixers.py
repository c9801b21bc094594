"""Throughput of mixer decoders at sizes that resemble a real model's layers, beside the closest other model at equal size
(Gidisun: the Qwen hybrid, DeltaNet + GQA with the same width, feed-forward, depth and vocabulary; Pezarax: Gidisun with the
same width, heads, depth and as many weights per token in its feed-forward; Zemozen: Pezarax with the same width, depth, number
of experts and weights per expert; Zarinex: Zemozen with the same width, depth, number of experts and weights per expert), and the time
of each design's kernels beside the like kernels of the other families.

    python -m pocketllm_b200.utils.bench_mixers --kernels [gidisun|pezarax|zemozen|zarinex]
    python bench.py --model gidisun|pezarax|zemozen|zarinex [--size 2k|4k]

Random weights; every weight set is larger than L2. Device times by CUDA events.
"""
from __future__ import annotations

import argparse
import json

import torch

from ..models import gidisun as gd
from ..models import pezarax as pz
from ..models import zarinex as zx
from ..models import zemozen as zm

VOCAB = 32000
#            width  ff     mLSTM (heads, dim, vdim)  GLA              latent (heads, dim, rot, vdim, rank, window)
SIZES = {"2k": (2048, 6144, (8, 128, 256), (16, 128, 128), (16, 128, 64, 128, 512, 1024)),
         "4k": (4096, 14336, (8, 256, 512), (16, 128, 256), (32, 128, 64, 128, 512, 1024))}
PATTERN = ("mlstm", "latent_attention", "gla", "gla", "mlstm", "latent_attention", "gla", "mlstm")


#                  width  retention (heads, dim, vdim)  attention (heads, kv heads, dim, vdim, chunk)  experts (number, top, ff)
PEZARAX_SIZES = {"2k": (2048, (16, 128, 128), (16, 4, 64, 128, 1024), (32, 2, 1536)),
                 "4k": (4096, (16, 128, 256), (32, 8, 64, 128, 1024), (32, 2, 3072))}
PEZARAX_PATTERN = ("retention", "attention", "retention", "retention", "retention", "attention", "retention", "retention")


def pezarax_config(size: str) -> pz.PezaraxConfig:
    W, r, a, e = PEZARAX_SIZES[size]
    decay = [1.0 - 2.0 ** (-5 - 8 * i / r[0]) for i in range(r[0])]
    mix = {"retention": {"heads": r[0], "dim": r[1], "vdim": r[2], "decay": decay, "rot": {"base": 1e4, "dims": r[1]}},
           "attention": {"heads": a[0], "kv_heads": a[1], "dim": a[2], "vdim": a[3], "scale": a[2] ** -0.5, "diff": 0.4, "mask": {"size": a[4]},
                         "rot": {"base": 5e5, "dims": a[2]}}}
    mlp = {"kind": "moe", "expert": {"ff": e[2]}, "router": {"experts": e[0], "top": e[1]}}
    return pz.PezaraxConfig.from_dict({"architecture": pz.ARCH, "vocab": VOCAB, "width": W, "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0}, "logit_scale": 0.5,
                                       "layers": [{"type": t, "mixer": mix[t], "mlp": mlp} for t in PEZARAX_PATTERN]})


#                  width  both attentions (heads, kv heads, dim, vdim, window)  state space (heads, vdim, state, groups)  experts (number, identities, top, ff)
ZEMOZEN_SIZES = {"2k": (2048, (16, 4, 128, 128, 1024), (32, 64, 128, 4), (32, 4, 2, 1024)),
                 "4k": (4096, (32, 8, 128, 128, 1024), (64, 64, 128, 8), (32, 4, 2, 2048))}
ZEMOZEN_PATTERN = ("parallel", "parallel", "attention", "parallel", "parallel", "parallel", "attention", "parallel")


def zemozen_config(size: str) -> zm.ZemozenConfig:
    W, a, s, e = ZEMOZEN_SIZES[size]
    att = {"heads": a[0], "kv_heads": a[1], "dim": a[2], "vdim": a[3], "scale": a[2] ** -0.5, "mask": {"size": a[4]}, "rot": {"base": 5e5, "dims": a[2]}}
    mix = {"attention": att | {"v_mix": True, "rot": att["rot"] | {"scaling": {"factor": 8.0}}},
           "parallel": {"left": att | {"softcap": 30.0}, "left_scale": 0.8, "right_scale": 0.9,
                        "right": {"heads": s[0], "vdim": s[1], "state": s[2], "groups": s[3], "conv": 4, "norm_groups": s[3]}}}
    mlp = {"kind": "moe", "expert": {"ff": e[3]}, "router": {"experts": e[0], "identity": e[1], "top": e[2]}}
    return zm.ZemozenConfig.from_dict({"architecture": zm.ARCH, "vocab": VOCAB, "width": W, "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0},
                                       "residual_mult": 0.7, "layers": [{"type": t, "mixer": mix[t], "mlp": mlp} for t in ZEMOZEN_PATTERN]})


#                  width  scan (inner, state, dt rank)  latent (heads, dim, vdim, query rank, rank)  HGRN2 (heads, dim, vdim)  experts (number, top, ff, shared ff)
ZARINEX_SIZES = {"2k": (2048, (4096, 16, 128), (16, 128, 128, 768, 512), (16, 128, 128), (32, 2, 1024, 1024)),
                 "4k": (4096, (8192, 16, 256), (32, 128, 128, 1536, 512), (32, 128, 128), (32, 2, 2048, 2048))}
ZARINEX_PATTERN = ("mamba1", "latent_attention", "mamba1", "hgrn2", "mamba1", "latent_attention", "hgrn2", "mamba1")


def zarinex_config(size: str) -> zx.ZarinexConfig:
    W, s, a, h, e = ZARINEX_SIZES[size]
    mix = {"mamba1": {"inner": s[0], "state": s[1], "dt_rank": s[2], "conv": 4},
           "latent_attention": {"heads": a[0], "dim": a[1], "vdim": a[2], "q_rank": a[3], "kv_rank": a[4], "scale": a[1] ** -0.5},
           "hgrn2": {"heads": h[0], "dim": h[1], "vdim": h[2]}}
    mlp = {"kind": "moe", "expert": {"ff": e[2]}, "router": {"experts": e[0], "top": e[1]}, "shared": {"ff": e[3]}}
    return zx.ZarinexConfig.from_dict({"architecture": zx.ARCH, "vocab": VOCAB, "width": W, "norm": {"eps": 1e-5}, "postln_alpha": 2.0,
                                       "layers": [{"type": t, "mixer": mix[t], "mlp": mlp} for t in ZARINEX_PATTERN]})


def config(size: str, ff: int | None = None) -> gd.GidisunConfig:
    W, dense_ff, m, g, a = SIZES[size]
    ff = ff or dense_ff
    mix = {"mlstm": {"heads": m[0], "dim": m[1], "vdim": m[2], "gate_cap": 12.0},
           "gla": {"heads": g[0], "dim": g[1], "vdim": g[2], "tau": 14.0},
           "latent_attention": {"heads": a[0], "dim": a[1], "rot_dim": a[2], "vdim": a[3], "kv_rank": a[4], "scale": (a[1] + a[2]) ** -0.5,
                                "mask": {"size": a[5]}, "rot": {"base": 5e5, "dims": a[2],
                                                                "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}}
    return gd.GidisunConfig.from_dict({"architecture": gd.ARCH, "vocab": VOCAB, "width": W, "norm": {"eps": 1e-5},
                                       "layers": [{"type": t, "mixer": mix[t], "mlp": {"kind": "dense", "ff": ff}} for t in PATTERN]})


def build(design: str, size: str, batch: int, context: int, ff: int | None = None):
    """(runtime with random weights, bytes of weights that one decoded token streams)."""
    from ..runtime.mixer_runtime import MixerRuntime
    mod, c = {"gidisun": lambda: (gd, config(size, ff)), "pezarax": lambda: (pz, pezarax_config(size)), "zemozen": lambda: (zm, zemozen_config(size)),
              "zarinex": lambda: (zx, zarinex_config(size))}[design]()
    t = mod.random_tensors(c, 0, device="cuda")
    pages = batch * (-(-context // 64))
    streamed = 0.0
    for n, v in t.items():
        share = 1.0
        if ".mlp.e" in n:
            L = c.layers[int(n[1:n.index(".")])]
            share = L.top / (L.experts + getattr(L, "identity", 0))
        streamed += v.numel() * 2 * share if n != "embed" or "head" not in t else 0.0
    rt = MixerRuntime(mod.build_model(c, t, slots=batch, pages=pages), max_requests=batch, pages=pages)
    return rt, streamed


def requests(rt, prompts, n: int, d: int, warmup: int, batch: int, clocks=None) -> dict:
    """Prefill and decode milliseconds of single requests, decode milliseconds of `batch` requests together, and end-to-end
    decode seconds with every token read back: sums over the prompts behind the first `warmup`."""
    import contextlib
    import time

    from ..runtime.mixer_runtime import StepEntry
    e0, e1, e2 = (torch.cuda.Event(enable_timing=True) for _ in range(3))

    def request(prompt, rids):
        e0.record()
        tok = [int(rt.step([StepEntry(r, prompt, (n - 1,))])[0].argmax()) for r in rids]
        e1.record()
        for a in range(0, d, rt.HIST):
            out = rt.decode_greedy(rids, tok, min(rt.HIST, d - a))
            tok = [o[-1] for o in out]
        e2.record()
        torch.cuda.synchronize()
        for r in rids:
            rt.release(r)
        return e0.elapsed_time(e1), e1.elapsed_time(e2)

    for p in prompts[:warmup]:
        request(p, [0])
        request(p, list(range(batch)))
    r = dict(prefill_ms=0.0, decode_ms=0.0, batch_ms=0.0, e2e_s=0.0)
    l0 = rt.launches
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    with clocks if clocks is not None else contextlib.nullcontext():
        for p in prompts[warmup:]:
            a, b = request(p, [0])
            r["prefill_ms"] += a
            r["decode_ms"] += b
        torch.cuda.synchronize()
    r.update(wall_ms=(time.perf_counter() - t0) * 1e3, launches=rt.launches - l0)
    for p in prompts[warmup:]:
        r["batch_ms"] += request(p, list(range(batch)))[1]
    # end to end through the step function: prompt ids from the host, every token read back as soon as its step ends
    for p in prompts[warmup:]:
        tok = int(rt.step([StepEntry(0, p, (n - 1,))])[0].argmax())
        torch.cuda.synchronize()
        w0 = time.perf_counter()
        for _ in range(d):
            tok = int(rt.step([StepEntry(0, [tok], (0,))])[0].argmax())
        r["e2e_s"] += time.perf_counter() - w0
        rt.release(0)
    rt.check_status()
    return r


def closest_to_pezarax(size: str, prompts, n: int, d: int, warmup: int, batch: int) -> dict:
    """Gidisun with a SwiGLU of as many weights per token as the chosen experts have."""
    _, _, _, (_, top, ff) = PEZARAX_SIZES[size]
    rt, streamed = build("gidisun", size, batch, n + d + 64, ff=2 * top * ff // 3)
    r, k = requests(rt, prompts, n, d, warmup, batch), len(prompts) - warmup
    return {"model": "Gidisun (mLSTM, GLA, latent attention, SwiGLU; bf16 weights)", "prefill_tok_s": round(k * n / r["prefill_ms"] * 1e3, 1),
            "decode_tok_s": round(k * d / r["decode_ms"] * 1e3, 1), "decode_tok_s_batch": round(k * d * batch / r["batch_ms"] * 1e3, 1),
            "weight_gb_per_token": round(streamed / 1e9, 2), "decode_weight_gbs": round(streamed * k * d / r["decode_ms"] / 1e6, 1)}


def closest_to_zemozen(size: str, prompts, n: int, d: int, warmup: int, batch: int) -> dict:
    """Pezarax with as many experts of as many weights."""
    rt, streamed = build("pezarax", size, batch, n + d + 64)
    r, k = requests(rt, prompts, n, d, warmup, batch), len(prompts) - warmup
    return {"model": "Pezarax (retention, differential attention, routed experts; bf16 weights)", "prefill_tok_s": round(k * n / r["prefill_ms"] * 1e3, 1),
            "decode_tok_s": round(k * d / r["decode_ms"] * 1e3, 1), "decode_tok_s_batch": round(k * d * batch / r["batch_ms"] * 1e3, 1),
            "weight_gb_per_token": round(streamed / 1e9, 2), "decode_weight_gbs": round(streamed * k * d / r["decode_ms"] / 1e6, 1)}


def closest_to_zarinex(size: str, prompts, n: int, d: int, warmup: int, batch: int) -> dict:
    """Zemozen with as many experts of as many weights."""
    rt, streamed = build("zemozen", size, batch, n + d + 64)
    r, k = requests(rt, prompts, n, d, warmup, batch), len(prompts) - warmup
    return {"model": "Zemozen (windowed attention beside a state-space recurrence, routed experts; bf16 weights)", "prefill_tok_s": round(k * n / r["prefill_ms"] * 1e3, 1),
            "decode_tok_s": round(k * d / r["decode_ms"] * 1e3, 1), "decode_tok_s_batch": round(k * d * batch / r["batch_ms"] * 1e3, 1),
            "weight_gb_per_token": round(streamed / 1e9, 2), "decode_weight_gbs": round(streamed * k * d / r["decode_ms"] / 1e6, 1)}


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
        self.ctx = StepContext(T, dev([0] * T), dev(p["pos"]), dev(p["slot"]), dev(p["last"]), dev(p["behind"]), table, Workspace("cuda"),
                               torch.zeros(1, dtype=torch.int32, device="cuda"), short=dev(p["short"]), n_short=len(p["short"]), rows=dev(p["rows"]),
                               n_rows=len(p["rows"]), all_rows=dev(range(T)), long=dev(p["long"]), n_long=len(p["long"]), chunks=dev(p["chunks"]),
                               chunk0=dev(p["chunk0"]), n_chunks=len(p["chunks"]), tiles=dev(p["tiles"]), n_tiles=len(p["tiles"]), tile0=dev(p["tile0"]),
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
    if kind == "retention":
        m = ml.RetentionMixer(w, {"heads": H, "dim": D, "vdim": V, "decay": [0.99] * H, "rot": {"base": 1e4, "dims": D}}, 1e-5, torch.bfloat16, "cuda", b.slots)
    elif kind == "mlstm":
        w.update({"i": r(H, W), "f": r(H, W), "i.b": torch.zeros(H), "f.b": torch.full((H,), 3.0), "norm": torch.ones(H * V)})
        m = ml.MLSTMMixer(w, {"heads": H, "dim": D, "vdim": V, "gate_cap": 12.0}, 1e-5, torch.bfloat16, "cuda", b.slots)
    elif kind == "hgrn2":
        w.update({"f": r(H * D, W), "f.b": torch.full((H * D,), 3.0), "lower": torch.full((H * D,), 0.3), "norm": torch.ones(V)})
        m = ml.HGRN2Mixer(w, {"heads": H, "dim": D, "vdim": V}, 1e-5, torch.bfloat16, "cuda", b.slots)
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


def _state_space(dims, T: int, singles: bool, dtype=torch.bfloat16):
    """The state-space recurrence of one layer with its convolution, gate and norm: (call, flops, bytes of states)."""
    from ..models import mixer_layers as ml
    from ..ops import mixer_ops as mo
    H, V, N, G = dims
    W, inner = 1024, dims[0] * dims[1]
    ch = inner + 2 * G * N
    b = _Batch(T, 4096, 64, singles=singles)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    w = {"in": r(2 * inner + 2 * G * N + H, W), "conv": r(ch, 4), "conv.b": torch.zeros(ch), "dt_bias": torch.full((H,), -3.0), "A_log": torch.zeros(H),
         "D": torch.ones(H), "norm": torch.ones(inner)}
    m = ml.StateSpaceMixer(w, {"heads": H, "vdim": V, "state": N, "groups": G, "conv": 4, "norm_groups": G}, 1e-5, dtype, "cuda", b.slots)
    m.at(0)
    p = ml.FusedLinear([("in", w["in"])], torch.bfloat16, "cuda")(b.ctx, torch.randn(T, W, device="cuda").to(torch.bfloat16), "proj", torch.float32)
    mix = b.ctx.ws.rows("mix", T, inner, dtype)

    def call():
        m.run(b.ctx, p, mix)
    call.keep = (m, b, p, mix)
    flops = 2.0 * T * (H * (2 * N * V + 32 * V) + G * 64 * N)       # states twice, weights of a chunk's earlier tokens (half of 64), products of a group
    return call, flops, T * H * N * V * 8.0 if singles else 0.0


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


def _paged(dims, T: int, start: int, singles: bool):
    """The attention of one differential layer after its input projection, without the output projection; returns
    {kernel: (call, flops, bytes)}. The descriptor holds bare addresses: every call keeps the tensors behind them alive."""
    from ..models import mixer_layers as ml
    from ..ops import mixer_ops as mo
    H, G, D, V, chunk = dims
    W, nq = 1024, 2 * dims[0]
    b = _Batch(T, start, start + T, singles=singles)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    m = ml.GroupedAttentionMixer({"q": r(nq * D, W), "k": r(2 * G * D, W), "v": r(G * V, W), "o": r(W, H * V), **{n: torch.zeros(D) for n in ("lq1", "lk1", "lq2", "lk2")}},
                                 {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": D ** -0.5, "diff": 0.4, "mask": {"size": chunk} if chunk else None,
                                  "rot": {"base": 1e4, "dims": D}}, 1e-5, torch.bfloat16, "cuda", b.pages, start + T, mask="chunk")
    m.cache.normal_()
    ctx, ws = b.ctx, b.ctx.ws
    p = m.proj(ctx, torch.randn(T, m.proj.K, device="cuda").to(torch.bfloat16), "proj", torch.float32)
    mix = ws.rows("mix", T, m.out.K, torch.bfloat16)
    d = m.describe(ctx, p, mix)
    see = lambda q: q + 1 - (q // chunk * chunk if chunk else 0)
    span = T * see(start) if singles else sum(see(start + i) for i in range(T))
    return _paged_calls(m, b, p, mix, d, T, span, singles)


def _windowed(dims, T: int, start: int, singles: bool, parallel: bool):
    """The same for one of Zemozen's attentions: mixed values and a gate per head, or capped scores and a sink."""
    from ..models import mixer_layers as ml
    H, G, D, V, window = dims
    W = 1024
    b = _Batch(T, start, start + T, singles=singles)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    w = {"q": r(H * D, W), "k": r(G * D, W), "v": r(G * V, W), "o": r(W, H * V), "q.norm": torch.ones(D), "k.norm": torch.ones(D)}
    c = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": D ** -0.5, "mask": {"size": window} if window else None, "rot": {"base": 1e4, "dims": D}}
    if parallel:
        m = ml.GroupedAttentionMixer(w, c | {"softcap": 30.0}, 1e-5, torch.bfloat16, "cuda", b.pages, start + T, neighbours=True, sink=0.0)
    else:
        w.update(g=r(H, W), vmix=torch.tensor(0.4))
        m = ml.GroupedAttentionMixer(w, c, 1e-5, torch.bfloat16, "cuda", b.pages, start + T, v_mix="mix")
    m.cache.normal_()
    p = m.proj(b.ctx, torch.randn(T, m.proj.K, device="cuda").to(torch.bfloat16), "proj", torch.float32)
    mix = b.ctx.ws.rows("mix", T, m.out.K, torch.bfloat16)
    see = lambda q: min(q + 1, window or 1 << 30)
    return _paged_calls(m, b, p, mix, m.describe(b.ctx, p, mix), T, T * see(start) if singles else sum(see(start + i) for i in range(T)), singles)


def _paged_calls(m, b, p, mix, d, T: int, span: int, singles: bool) -> dict:
    from ..ops import mixer_ops as mo
    ctx, ws, nq, D, V = b.ctx, b.ctx.ws, m.H * m.maps, m.D, m.V
    keep = (m, b, p, mix)
    flops = 2.0 * span * nq * (D + V)
    if singles:
        d.nsplit = m.nsplit
        po, pm = ws.flat("po", T * m.nsplit * nq * V, torch.float32), ws.flat("pm", T * m.nsplit * nq * 2, torch.float32)
        qx = ws.flat("qx", T * nq * D, torch.float32)
        d.qx, d.part_o, d.part_ml = qx.data_ptr(), po.data_ptr(), pm.data_ptr()
        return {"prep": (lambda k=keep: mo.paged_prep(d, T), 0, 0), "rows": (lambda k=(keep, po, pm, qx): mo.paged_rows(d, ctx.rows, T), flops, span * m.row * 2.0),
                "merge": (lambda k=(keep, po, pm): mo.paged_merge(d, ctx.rows, T), 0, T * m.nsplit * nq * V * 4.0)}
    qf = ws.flat("qf", T * nq * m.q_ld, torch.bfloat16)
    d.qf = qf.data_ptr()
    return {"prep": (lambda k=keep: mo.paged_prep(d, T), 0, T * (p.shape[1] * 4.0 + m.row * 2 + nq * m.q_ld * 2)),
            "attention": (lambda k=(keep, qf): mo.paged_prefill(d, T, b.pages, ctx.tiles, ctx.n_tiles, ctx.long), flops, 0)}


def _experts(W: int, E: int, top: int, ff: int, T: int, sets: int, identity: int | None = None):
    """Routed experts of `sets` layers (together larger than L2): {kernel: (call over all layers, flops, bytes)} per layer.
    `identity`: gated experts, behind them as many identities."""
    from ..models import mixer_layers as ml
    from ..ops import mixer_ops as mo
    ctx = ml.StepContext(T, *[None] * 6, ml.Workspace("cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"))
    g = torch.Generator(device="cuda").manual_seed(0)
    r = lambda *s: (torch.randn(*s, generator=g, device="cuda") * s[-1] ** -0.5).to(torch.bfloat16)
    gated = identity is not None
    rows = lambda: [r(ff, W) for _ in range(E)]
    if gated:
        router = mo.Router(E, top, score="softmax", renorm=True, on_output=True, identity=identity)
        new = lambda: ml.RoutedExperts(r(router.outputs, W), rows(), [r(W, ff) for _ in range(E)], router, torch.bfloat16, "cuda", gate=rows(),
                                       correction=torch.zeros(router.outputs))
    else:
        new = lambda: ml.RoutedExperts(r(E, W), rows(), [r(W, ff) for _ in range(E)], mo.Router(E, top), torch.bfloat16, "cuda")
    layers = [new() for _ in range(sets)]
    h = torch.randn(T, layers[0].up.shape[2], generator=g, device="cuda").to(torch.bfloat16)
    R, ws = T * top, ctx.ws
    z = [m.router(ctx, h, f"router{i}", torch.float32) for i, m in enumerate(layers)]
    n = E + (identity or 0)
    used = E * (1.0 - (1.0 - top / n) ** T)                            # experts that are expected to be used
    flops, nbytes = 2.0 * R * E / n * W * ff, used * W * ff * 2.0      # of the down product
    up = 2 if gated else 1
    kw = lambda m: {"correction": m.correction, "skip_w": ws.flat("skip", T, torch.float32)} if gated else {}
    ids, hidden = ws.flat("ids", R, torch.int32), ws.rows("hid", R, layers[0].ff, torch.bfloat16)
    keep = (layers, z)
    out = {"whole layer with router": (lambda k=keep: [m.forward(ctx, h) for m in layers], (up + 1) * flops, (up + 1) * nbytes)}
    if T <= mo.ROWS_MAX:
        y = ws.rows("yy", T, layers[0].down.shape[1], torch.float32)
        out["up rows (choice included)"] = (lambda: [mo.expert_up_rows(m.route, q, h, m.up, ids, hidden, gated=gated, **kw(m)) for m, q in zip(layers, z)],
                                           up * flops, up * nbytes)
        out["down rows"] = (lambda: [mo.expert_down_rows(m.route, ids, hidden, m.down, W, y) for m in layers], flops, nbytes)
        return out
    place, seg, sc = ws.rows("pl", T, top, torch.int32), ws.flat("sg", E + 1, torch.int32), ws.flat("sc", R, torch.float32)
    x, y, rw = ws.rows("rx", R, h.shape[1], torch.bfloat16), ws.rows("yy", R, layers[0].down.shape[1], torch.float32), ws.flat("rw", R, torch.float32)
    group = lambda m, q: mo.expert_group(m.route, q, h, ids, rw, seg, place, sc, x, **kw(m))
    group(layers[0], z[0])
    out["choice, grouping, gather"] = (lambda: [group(m, q) for m, q in zip(layers, z)], 0, T * W * 2.0 + R * W * 2.0)
    group(layers[0], z[0])
    out["up (grouped GEMM, SwiGLU)" if gated else "up (grouped GEMM, squared ReLU)"] = (
        lambda: [mo.grouped_linear(x, m.up, seg, hidden, ctx.status, relu2=not gated, swiglu=gated, row_scale=sc, scale_after=gated) for m in layers],
        up * flops, up * nbytes)
    out["down (grouped GEMM, fp32 out)"] = (lambda: [mo.grouped_linear(hidden, m.down, seg, y, ctx.status) for m in layers], flops, nbytes)
    return out


def pezarax_kernels() -> None:
    from .. import ops
    from ..ops import mixer_ops as mo
    from . import bench_kernels as bk
    show = lambda name, d, **kw: print(json.dumps({"kernel": name, **kw, **d}), flush=True)
    dims = (16, 128, 256)
    for T in (512, 2048):
        for kind in ("retention", "gla"):
            f, fl, _ = _state(kind, dims, T, False)
            show(f"{kind} chunk form + head norm", _roof(timed(f), fl), T=T, dims=dims)
        r = bk.bench_deltanet(T, 16, 32, 20)
        show("like kernel: chunked DeltaNet", _roof(r["us"], 2.0 * T * 32 * (3 * 128 * 128 + 2.5 * 64 * 128 + 64 * 64 * 1.0)), T=T)
    for B in (1, 8):
        for kind in ("retention", "gla"):
            f, _, nb = _state(kind, dims, B, True)
            show(f"{kind} rows form + head norm", _roof(timed(f), 0, nb), B=B, dims=dims)
    for dims in ((32, 8, 64, 128, 0), (32, 8, 64, 128, 1024), (32, 8, 128, 128, 0)):
        for k, (f, fl, nb) in _paged(dims, 512, 8192 - 512, False).items():
            show("differential prefill: " + k, _roof(timed(f), fl, nb), T=512, context=8192, dims=dims)
    show("like kernel: GQA prefill", bk.bench_attention(512, 8192, 32, 8, 20))
    f, fl, nb = _latent((32, 128, 64, 128, 512, 1024), 512, 8192 - 512, False)["prep"]
    show("like kernel: latent prep", _roof(timed(f), fl, nb), T=512)
    for B, chunk in ((1, 1024), (8, 1024), (1, 0), (8, 0)):
        start = 8191
        for k, (f, fl, nb) in _paged((32, 8, 64, 128, chunk), B, start, True).items():
            show("differential rows: " + k, _roof(timed(f), fl, nb), B=B, context=start + 1, chunk=chunk)
    for B in (1, 8):
        for ctx in (1024, 8192):
            q = torch.randn(B, 32, 128, device="cuda").to(torch.bfloat16)
            kc, vc = (torch.randn(8, ctx, 128, device="cuda").to(torch.bfloat16) for _ in range(2))
            pos = torch.full((B,), ctx - 1, device="cuda", dtype=torch.int32)
            ns = max(1, min(32, ctx // 64))
            us = timed(lambda: ops.gqa_decode(q, kc, vc, pos, nsplit=ns))
            show("like kernel: GQA decode rows", _roof(us, 4.0 * B * 32 * 128 * ctx, B * ctx * 8 * 256 * 2.0), B=B, context=ctx, nsplit=ns)
    W, E, top, ff = 4096, 32, 2, 3072
    for T in (1, 8, 64, 512, 2048):
        sets = 2
        for k, (f, fl, nb) in _experts(W, E, top, ff, T, sets).items():
            us = timed(f, reps=8) / sets
            show("experts: " + k, _roof(us, fl, nb), T=T)
    for M in (1, 2, 8):
        for N, K in ((ff * 2, W), (W, ff * 2)):
            ws = [torch.randn(N, K, device="cuda").to(torch.bfloat16) for _ in range(max(2, -(-(300 << 20) // (N * K * 2))))]
            x, y, s = torch.randn(M, K, device="cuda").to(torch.bfloat16), torch.empty(M, N, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
            us = timed(lambda: [mo.linear(x, w, y, s) for w in ws], reps=8) / len(ws)
            show("like kernel: few-row linear", _roof(us, 0, N * K * 2.0), M=M, N=N, K=K)
    from ctypes import c_int, c_void_p
    for T in (64, 512, 2048):
        R = T * top
        seg = torch.linspace(0, R, E + 1, device="cuda").to(torch.int32)
        a = torch.randn(R, W, device="cuda").to(torch.bfloat16)
        w = torch.randn(E * 2 * ff // 2, W, device="cuda").to(torch.bfloat16)
        c, s = torch.empty(R, ff // 2, device="cuda", dtype=torch.bfloat16), torch.zeros(1, dtype=torch.int32, device="cuda")
        K = ops.lib.kernels()
        ptr = lambda t: c_void_p(t.data_ptr())
        call = lambda: K.pk_gemm_bf16_grouped(ptr(a), c_int(W), ptr(w), ptr(seg), c_int(E), c_int(R), c_int(ff), c_int(W), c_int(1), ptr(c), c_int(ff // 2), ptr(s),
                                              c_int(mo.sm_count()), c_void_p(torch.cuda.current_stream().cuda_stream))
        show("like kernel: grouped GEMM, SwiGLU", _roof(timed(call), 2.0 * R * W * ff, E * W * ff * 2.0), T=T)
    for T in (1, 2048):
        x, y, w = torch.randn(T, 4096, device="cuda"), torch.randn(2 * T, 4096, device="cuda"), torch.randn(4096, device="cuda")
        place = torch.randperm(2 * T, device="cuda").to(torch.int32).view(T, 2)
        o = torch.empty(T, 4096, device="cuda", dtype=torch.bfloat16)
        show("residual add + norm", _roof(timed(lambda: mo.sandwich_norm(x, y=y, w_pre=w, out=o, eps=1e-5)), 0, T * 4096 * 14.0), T=T)
        show("sum of two expert rows + residual add + norm", _roof(timed(lambda: mo.sandwich_norm(x, y=y, y_rows=place, w_pre=w, out=o, eps=1e-5)), 0, T * 4096 * 18.0), T=T)
        show("like kernel: two norms + residual add", _roof(timed(lambda: mo.sandwich_norm(x, y=y, w_post=w, w_pre=w, out=o, eps=1e-5)), 0, T * 4096 * 14.0), T=T)


def zemozen_kernels() -> None:
    """The new kernels and variants, each followed by the like kernel of Pezarax in the same run."""
    from ..ops import mixer_ops as mo
    show = lambda name, d, **kw: print(json.dumps({"kernel": name, **kw, **d}), flush=True)
    space, ret = (64, 64, 128, 8), (16, 128, 256)
    for T in (512, 2048):
        for dt in (torch.bfloat16, torch.float32):
            f, fl, _ = _state_space(space, T, False, dt)
            show("state space prefill, " + ("tensor cores" if dt == torch.bfloat16 else "fp32") + " (convolution, gate, norm included)", _roof(timed(f), fl), T=T,
                 dims=space)
        f, fl, _ = _state("retention", ret, T, False)
        show("like kernel: retention chunk form + head norm", _roof(timed(f), fl), T=T, dims=ret)
    for B in (1, 8):
        f, _, nb = _state_space(space, B, True)
        show("state space rows form (convolution, gate, norm included)", _roof(timed(f), 0, nb), B=B, dims=space)
        f, _, nb = _state("retention", ret, B, True)
        show("like kernel: retention rows form + head norm", _roof(timed(f), 0, nb), B=B, dims=ret)
    for T in (512, 2048):
        for window in (0, 1024):
            for par in (False, True):
                for k, (f, fl, nb) in _windowed((32, 8, 128, 128, window), T, 8192 - T, False, par).items():
                    show(("capped" if par else "gated") + " prefill: " + k, _roof(timed(f), fl, nb), T=T, context=8192, window=window)
            for k, (f, fl, nb) in _paged((32, 8, 64, 128, window), T, 8192 - T, False).items():
                show("like kernel: differential prefill: " + k, _roof(timed(f), fl, nb), T=T, context=8192, chunk=window)
    for B in (1, 8):
        for window in (1024, 0):
            for par in (False, True):
                for k, (f, fl, nb) in _windowed((32, 8, 128, 128, window), B, 8191, True, par).items():
                    show(("capped" if par else "gated") + " rows: " + k, _roof(timed(f), fl, nb), B=B, context=8192, window=window)
            for k, (f, fl, nb) in _paged((32, 8, 64, 128, window), B, 8191, True).items():
                show("like kernel: differential rows: " + k, _roof(timed(f), fl, nb), B=B, context=8192, chunk=window)
    W, E, top = 4096, 32, 2
    for T in (1, 8, 64, 512, 2048):
        for name, ff, ident in (("gated experts: ", 2048, 4), ("like kernel: experts: ", 3072, None)):
            for k, (f, fl, nb) in _experts(W, E, top, ff, T, 2, ident).items():
                show(name + k, _roof(timed(f, reps=8) / 2, fl, nb), T=T)
    for T in (1, 2048):
        x, y, w = torch.randn(T, 4096, device="cuda"), torch.randn(2 * T, 4096, device="cuda"), torch.randn(4096, device="cuda")
        place = torch.randperm(2 * T, device="cuda").to(torch.int32).view(T, 2)
        o, sw = torch.empty(T, 4096, device="cuda", dtype=torch.bfloat16), torch.rand(T, device="cuda")
        f = lambda: mo.sandwich_norm(x, y=y, y_rows=place, y_scale=0.7, skip=o, skip_w=sw, w_pre=w, out=o, eps=1e-5)
        show("expert rows + identity + residual add + norm", _roof(timed(f), 0, T * 4096 * 20.0), T=T)
        show("like kernel: sum of two expert rows + residual add + norm", _roof(timed(lambda: mo.sandwich_norm(x, y=y, y_rows=place, w_pre=w, out=o, eps=1e-5)), 0,
                                                                               T * 4096 * 18.0), T=T)


def _selective_scan(dims, T: int, singles: bool, dtype=torch.bfloat16) -> dict:
    """One selective-scan layer between its input and output projections: {kernel: (call, flops, bytes)}. Flops of the recurrence: two
    products, a decay and two sums per channel and state."""
    from ..models import mixer_layers as ml
    from ..ops import mixer_ops as mo
    inner, N, rank = dims
    W, es = 64, 2 if dtype == torch.bfloat16 else 4
    b = _Batch(T, 4096, 64, singles=singles)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    w = {"in": r(2 * inner, W), "conv": r(inner, 4), "conv.b": torch.zeros(inner), "x": r(rank + 2 * N, inner), "dt": r(inner, rank), "dt.b": torch.full((inner,), -3.0),
         "A_log": torch.log(torch.arange(1, N + 1).float()).repeat(inner, 1), "D": torch.ones(inner), "o": r(W, inner)}
    m = ml.SelectiveScanMixer(w, {"inner": inner, "state": N, "dt_rank": rank, "conv": 4}, 1e-5, dtype, "cuda", b.slots)
    ctx, ws = b.ctx, b.ctx.ws
    p = m.proj(ctx, torch.randn(T, W, device="cuda").to(dtype), "proj", torch.float32)
    mix = ws.rows("mix", T, m.out.K, dtype)
    m.run(ctx, p, mix)
    x, dbc = ws.rows("scan_x", T, m.dbc.K, dtype), ws.rows("scan_dbc", T, m.dbc.N, torch.float32)
    d = mo.SelectiveScan(proj=p.data_ptr(), ld=p.stride(0), xc=x.data_ptr(), ldx=x.stride(0), out=mix.data_ptr(), ldo=mix.stride(0), pos=ctx.pos.data_ptr(),
                         slot=ctx.slot.data_ptr(), dbc=dbc.data_ptr(), ldb=dbc.stride(0), **m.desc)
    keep = (m, b, p, mix, x, dbc)
    flops = 5.0 * T * inner * N
    out = {"all between the projections": (lambda k=keep: m.run(ctx, p, mix), 0, 0),
           "convolution": (lambda k=keep: mo.scan_conv(d, T), 0, T * inner * (4.0 + es))}
    if singles:
        out["rows form (step sizes, gate included)"] = (lambda k=keep: mo.scan_rows(d, ctx.short, ctx.n_short), 0, T * inner * N * 8.0 + inner * (m.dt.K // 2 * es + N * 4))
        return out
    terms, dt = ws.rows("scan_d", T, m.dt.K, dtype), ws.rows("scan_dt", T, m.dt.N, torch.float32)
    d.dt, d.ldt = dt.data_ptr(), dt.stride(0)
    if dtype == torch.bfloat16:
        out["step sizes (split and product)"] = (lambda k=(keep, terms): (mo.scan_split(dbc, m.rank, terms), m.dt(ctx, terms, "scan_dt", torch.float32)),
                                                 2.0 * T * inner * m.dt.K, T * inner * 4.0)
    out["recurrence (gate included)"] = (lambda k=(keep, dt): mo.scan_tiles(d, ctx.long, ctx.n_long), flops, T * inner * (8.0 + 2 * es))
    return out


def _gated_latent(dims, T: int, start: int, singles: bool):
    """Latent attention with queries from a latent and gated outputs, as `_latent`."""
    from ..models import mixer_layers as ml
    from ..ops import mixer_ops as mo
    H, D, V, Q, K = dims
    W = 64
    b = _Batch(T, start, start + T, singles=singles)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g) * s[-1] ** -0.5
    m = ml.LatentAttentionMixer({"dq": r(Q, W), "dq.norm": torch.ones(Q), "uq": r(H * D, Q), "dkv": r(K, W), "dkv.norm": torch.ones(K), "uk": r(H * D, K),
                                 "uv": r(H * V, K), "g": r(H * V, W), "o": r(W, H * V)},
                                {"heads": H, "dim": D, "vdim": V, "kv_rank": K, "scale": D ** -0.5}, 1e-5, torch.bfloat16, "cuda", b.pages, start + T)
    m.cache.normal_()
    ctx, ws = b.ctx, b.ctx.ws
    p = m.proj(ctx, torch.randn(T, m.proj.K, device="cuda").to(torch.bfloat16), "proj", torch.float32)
    at, qw = m.proj.at, m.qk_panels * 64
    gate, ql, mix = p[:, at["g"]:], ws.rows("lat_q", T, m.uq.K, torch.bfloat16), ws.rows("mix", T, m.out.K, torch.bfloat16)
    span = sum(start + i + 1 for i in range(T)) if not singles else T * (start + 1)
    prep = lambda k=(m, b, p): mo.latent_prep(p, at["dq"], at["dkv"], H, D, 0, K, m.c_norm, 1e-5, m.freq, 1.0, ctx.pos, ctx.slot, m.cache, ctx.table, None, None, 0,
                                              q_rank=Q, q_norm=m.q_norm, ql=ql)
    prep_bytes = T * ((Q + K) * 4.0 + (m.row + m.uq.K) * 2)
    if singles:
        q, qx = m.uq(ctx, ql, "q_rows", torch.float32), ws.flat("qx", T * H * m.row, torch.float32)
        po, pm = ws.flat("po", T * m.nsplit * H * K, torch.float32), ws.flat("pm", T * m.nsplit * H * 2, torch.float32)
        return {"prep": (prep, 0, prep_bytes),
                "absorb": (lambda: mo.latent_absorb(q, 0, H, D, qw - D, K, m.uk, ctx.rows, T, qx, m.row, m.row), 2.0 * T * H * D * K, H * D * K * 2.0),
                "rows": (lambda: mo.latent_rows(qx, ctx.rows, T, ctx.pos, ctx.slot, m.cache, ctx.table, H, K, 0, m.scale, m.nsplit, po, pm),
                         2.0 * span * H * (m.row + K), span * m.row * 2.0),
                "merge + values + gate": (lambda: mo.latent_out(po, pm, m.nsplit, H, K, V, None, ctx.rows, T, m.uv, mix, gate), 2.0 * T * H * V * K, H * V * K * 2.0)}
    qf = m.uq(ctx, ql, "qf", torch.bfloat16)
    gather, total, longest = ctx.gather[0]
    c, kv = ws.rows("c", total, m.row, torch.bfloat16), ws.rows("kv", total, m.kv_w.shape[0], torch.bfloat16)
    return {"prep": (prep, 0, prep_bytes),
            "gather": (lambda: mo.latent_gather(m.cache, ctx.table, ctx.long, gather, 1, longest, c), 0, total * m.row * 4.0),
            "expand": (lambda: mo.linear(c, m.kv_w, kv, ctx.status), 2.0 * total * m.row * kv.shape[1], 0),
            "attention": (lambda: mo.latent_prefill(qf, T, kv, total, ctx.tiles, ctx.n_tiles, ctx.long, gather, H, m.qk_panels, m.v_panels, V, 0, m.scale, None, mix,
                                                    ctx.status, gate), 2.0 * span * H * (D + V), 0)}


def zarinex_kernels() -> None:
    """The new kernels and variants, each followed by the like kernel of Zemozen or Gidisun in the same run."""
    from ..ops import mixer_ops as mo
    show = lambda name, d, **kw: print(json.dumps({"kernel": name, **kw, **d}), flush=True)
    dims, space = (8192, 16, 256), (64, 64, 128, 8)
    for T in (512, 2048):
        for k, (f, fl, nb) in _selective_scan(dims, T, False).items():
            show("selective scan: " + k, _roof(timed(f), fl, nb), T=T, dims=dims)
        for k, (f, fl, nb) in _selective_scan(dims, T, False, torch.float32).items():
            show("selective scan, fp32: " + k, _roof(timed(f), fl, nb), T=T, dims=dims)
        f, fl, _ = _state_space(space, T, False)
        show("like kernel: state space prefill, tensor cores", _roof(timed(f), fl), T=T, dims=space)
    for B in (1, 8):
        for k, (f, fl, nb) in _selective_scan(dims, B, True).items():
            show("selective scan: " + k, _roof(timed(f), fl, nb), B=B, dims=dims)
        f, _, nb = _state_space(space, B, True)
        show("like kernel: state space rows form", _roof(timed(f), 0, nb), B=B, dims=space)
    head = (32, 128, 128)
    for T in (512, 2048):
        for kind in ("hgrn2", "gla"):
            f, fl, _ = _state(kind, head, T, False)
            show(("like kernel: " if kind == "gla" else "") + f"{kind} chunk form + head norm", _roof(timed(f), fl), T=T, dims=head)
    for B in (1, 8):
        for kind in ("hgrn2", "gla"):
            f, _, nb = _state(kind, head, B, True)
            show(("like kernel: " if kind == "gla" else "") + f"{kind} rows form + head norm", _roof(timed(f), 0, nb), B=B, dims=head)
    for T in (512, 2048):
        for k, (f, fl, nb) in _gated_latent((32, 128, 128, 1536, 512), T, 8192 - T, False).items():
            show("gated latent prefill: " + k, _roof(timed(f), fl, nb), T=T, context=8192)
        for k, (f, fl, nb) in _latent((32, 128, 64, 128, 512, 0), T, 8192 - T, False).items():
            show("like kernel: latent prefill: " + k, _roof(timed(f), fl, nb), T=T, context=8192)
    for B in (1, 8):
        for k, (f, fl, nb) in _gated_latent((32, 128, 128, 1536, 512), B, 1500, True).items():
            show("gated latent rows: " + k, _roof(timed(f), fl, nb), B=B)
        for k, (f, fl, nb) in _latent((32, 128, 64, 128, 512, 0), B, 1500, True).items():
            show("like kernel: latent rows: " + k, _roof(timed(f), fl, nb), B=B)
    W = 4096
    for T in (1, 8, 512, 2048):
        x, y, w = torch.randn(T, W, device="cuda"), torch.randn(2 * T, W, device="cuda"), torch.randn(W, device="cuda")
        xo, gate, y2, before = torch.empty_like(x), torch.randn(T, W, device="cuda"), torch.randn(T, W, device="cuda"), torch.randn(T, W, device="cuda")
        o, o2 = (torch.empty(T, W, device="cuda", dtype=torch.bfloat16) for _ in range(2))
        place = torch.randperm(2 * T, device="cuda").to(torch.int32).view(T, 2)
        b = _Batch(T, 64, 64, singles=T <= mo.ROWS_MAX).ctx
        base = dict(x=x, x_out=xo, gate=gate, ldg=W, gate_b=w, w=w, y=y, ldy=W, pos=b.pos, slot=b.slot, behind=b.behind, M=T, width=W, ldo=W, alpha=2.0, eps=1e-5, out=o)
        other = dict(shift=w, before=before, out_shift=o2)
        call = lambda **kw: mo.post_norm(mo.PostNorm(**{k: v.data_ptr() if isinstance(v, torch.Tensor) else v for k, v in (base | kw).items()}))
        show("gate + sum + norm, input kept", _roof(timed(lambda: call(save=before)), 0, T * W * 18.0), T=T)
        show("expert rows + shared expert + gate + sum + norm + token shift", _roof(timed(lambda: call(y_rows=place, y_top=2, y2=y2, ldy2=W, **other)),
                                                                                   0, T * W * 28.0), T=T)
        show("like kernel: residual add + norm", _roof(timed(lambda: mo.sandwich_norm(x, y=y, w_pre=w, out=o, eps=1e-5)), 0, T * W * 14.0), T=T)
        show("like kernel: sum of two expert rows + residual add + norm", _roof(timed(lambda: mo.sandwich_norm(x, y=y, y_rows=place, w_pre=w, out=o, eps=1e-5)), 0, T * W * 18.0), T=T)
    for M in (1, 8):
        for N, split in ((20480, 4096), (12288, 4096)):
            ws = [torch.randn(N, W, device="cuda").to(torch.bfloat16) for _ in range(3)]
            x, x2 = (torch.randn(M, W, device="cuda").to(torch.bfloat16) for _ in range(2))
            y, s = torch.empty(M, N, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
            show("few-row linear with two inputs", _roof(timed(lambda: [mo.linear2(x, x2, split, w, y, s) for w in ws], reps=8) / 3, 0, N * W * 2.0), M=M, N=N)
            show("like kernel: few-row linear", _roof(timed(lambda: [mo.linear(x, w, y, s) for w in ws], reps=8) / 3, 0, N * W * 2.0), M=M, N=N)


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--kernels", nargs="?", const="gidisun", choices=["gidisun", "pezarax", "zemozen", "zarinex"], help="time the design's kernels beside the like kernels")
    ap.add_argument("--size", default="2k", choices=sorted(SIZES))
    args = ap.parse_args()
    if args.kernels:
        {"gidisun": kernels, "pezarax": pezarax_kernels, "zemozen": zemozen_kernels, "zarinex": zarinex_kernels}[args.kernels]()
    else:
        print(json.dumps(closest_model(args.size, 512, 64, 3)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
