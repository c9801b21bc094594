"""Layers of decoders that are put together from mixers: every layer names its kind of mixer (recurrent state or attention)
and optionally a feed-forward, with its own sizes. The classes here hold a layer's weights in the layout of the kernels,
the device memory of its state or cache, and its forward pass over a mixed batch (`StepContext`): portions of prompts
beside single decoded tokens, any request in any slot.

Two precisions: bfloat16 (bf16 weights, activations and cache, fp32 accumulation; norms, gates, recurrences, attention
scores and the residual stream in fp32) and float32 (everything, without reduced-precision tensor modes).
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field

import torch

from ..ops import mixer_ops as mo


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class Workspace:
    """Named scratch buffers that only grow. A buffer that was outgrown stays alive: a captured graph may still point at it."""

    def __init__(self, device):
        self.device = torch.device(device)
        self._buf: dict[tuple[str, torch.dtype], torch.Tensor] = {}
        self._retired: list[torch.Tensor] = []

    def flat(self, name: str, numel: int, dtype: torch.dtype) -> torch.Tensor:
        b = self._buf.get((name, dtype))
        if b is None or b.numel() < numel:
            if b is not None:
                self._retired.append(b)
            b = self._buf[(name, dtype)] = torch.zeros(max(numel, 64), dtype=dtype, device=self.device)
        return b

    def rows(self, name: str, rows: int, cols: int, dtype: torch.dtype) -> torch.Tensor:
        return self.flat(name, rows * cols, dtype)[:rows * cols].view(rows, cols)

    def trim(self) -> None:
        self._retired.clear()


@dataclass
class StepContext:
    """One batch, as the kernels see it (int32 device tensors; a sequence is {first row, tokens, slot, first position})."""
    T: int
    tokens: torch.Tensor
    pos: torch.Tensor
    slot: torch.Tensor
    last_slot: torch.Tensor             # slot of the portion that ends at a row, else -1
    table: torch.Tensor                 # page table
    ws: Workspace
    status: torch.Tensor
    short: torch.Tensor | None = None   # portions of up to ROWS_MAX tokens
    n_short: int = 0
    rows: torch.Tensor | None = None    # rows that attend one by one
    n_rows: int = 0
    all_rows: torch.Tensor | None = None
    long: torch.Tensor | None = None
    n_long: int = 0
    chunks: torch.Tensor | None = None  # {first row, tokens, sequence, chunk of the sequence}
    chunk0: torch.Tensor | None = None
    n_chunks: int = 0
    tiles: torch.Tensor | None = None   # {first row, rows, sequence, 0}: up to 128 query rows of a long portion
    n_tiles: int = 0
    gather: dict = field(default_factory=dict)   # window -> ({first key row, its position} per long sequence, key rows, longest)


class FusedLinear:
    """Row blocks of several matrices that share their input as one [N, K] matrix, padded with zeros to what the kernels
    take; `at[name]` is the first output column of a block."""

    def __init__(self, blocks: list[tuple[str, torch.Tensor]], dtype: torch.dtype, device, k_pad: int | None = None):
        K = blocks[0][1].shape[1]
        self.K = k_pad or pad_to(K, 64)
        self.at, n = {}, 0
        for name, w in blocks:
            if w.shape[1] != K:
                raise ValueError(f"{name}: {w.shape[1]} input columns, the others have {K}")
            self.at[name] = n
            n += w.shape[0]
        self.N = pad_to(n, 8)
        w = torch.zeros(self.N, self.K, dtype=dtype)
        for name, b in blocks:
            w[self.at[name]:self.at[name] + b.shape[0], :K] = b.to(dtype)
        self.w = w.to(device)

    def __call__(self, ctx: StepContext, x: torch.Tensor, name: str, dtype: torch.dtype) -> torch.Tensor:
        out = ctx.ws.rows(name, x.shape[0], self.N, dtype)
        return mo.linear(x, self.w, out, ctx.status)


def _f32(t: torch.Tensor, device) -> torch.Tensor:
    return t.float().contiguous().to(device)


class RecurrentMixer:
    """Base of the mixers with an outer-product state per head. Subclasses fill `self.desc` with what is theirs."""
    per_head_norm = False

    def __init__(self, kind: int, w: dict, extra: list[str], heads: int, dim: int, vdim: int, eps: float, dtype, device, slots: int):
        if dim > 512:
            raise ValueError("recurrent mixers take key dims up to 512")
        self.H, self.D, self.V, self.eps, self.dtype = heads, dim, vdim, eps, dtype
        for n, r in (("q", heads * dim), ("k", heads * dim), ("v", heads * vdim), ("g", heads * vdim)):
            if w[n].shape[0] != r:
                raise ValueError(f"{n}: {w[n].shape[0]} rows, expected {r}")
        self.proj = FusedLinear([(n, w[n]) for n in ["q", "k", "v", "g"] + extra], dtype, device)
        self.out = FusedLinear([("o", w["o"])], dtype, device)
        self.norm = _f32(w["norm"], device)
        self.S = torch.zeros(slots, heads, dim, vdim, device=device)
        self.N = self.Ms = None
        a = self.proj.at
        self.keep: list[torch.Tensor] = []
        self.desc = dict(kind=kind, H=heads, D=dim, V=vdim, oq=a["q"], ok=a["k"], ov=a["v"], og=a["g"], qscale=dim ** -0.5, S=self.S.data_ptr())

    def state_bytes(self) -> int:
        return sum(t.numel() * 4 for t in (self.S, self.N, self.Ms) if t is not None)

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        T, ws = ctx.T, ctx.ws
        p = self.proj(ctx, h, "proj", torch.float32)
        o = ws.flat("raw_o", T * self.H * self.V, torch.float32)
        nq, m = ws.flat("raw_nq", T * self.H, torch.float32), ws.flat("raw_m", T * self.H, torch.float32)
        d = mo.StateMixer(proj=p.data_ptr(), ld=p.stride(0), o=o.data_ptr(), nq=nq.data_ptr(), m=m.data_ptr(), **self.desc)
        if ctx.n_short:
            mo.state_rows(d, ctx.short, ctx.n_short)
        if ctx.n_long:
            scratch = ws.flat("state_chunks", mo.state_chunk_workspace(d, ctx.n_chunks), torch.float32)
            mo.state_chunks(d, ctx.long, ctx.n_long, ctx.chunks, ctx.chunk0, ctx.n_chunks, scratch)
        mix = ws.rows("mix", T, self.out.K, self.dtype)
        mo.state_out(d, self.norm, self.per_head_norm, self.eps, ctx.last_slot, T, mix)
        return self.out(ctx, mix, "y", torch.float32)


class MLSTMMixer(RecurrentMixer):
    """Matrix memory of xLSTM with soft-capped exponential gates and a running maximum that starts at 0; the head outputs
    are normed with one weight over all heads and gated with a sigmoid."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, slots: int):
        super().__init__(mo.KIND_MLSTM, w, ["i", "f"], m["heads"], m["dim"], m["vdim"], eps, dtype, device, slots)
        self.N = torch.zeros(slots, self.H, self.D, device=device)
        self.Ms = torch.zeros(slots, self.H, device=device)
        bi, bf = _f32(w["i.b"], device), _f32(w["f.b"], device)
        self.keep += [bi, bf]
        a = self.proj.at
        self.desc.update(oi=a["i"], of=a["f"], bi=bi.data_ptr(), bf=bf.data_ptr(), cap=float(m["gate_cap"]), N=self.N.data_ptr(), Ms=self.Ms.data_ptr())


class GLAMixer(RecurrentMixer):
    """Gated linear attention: a decay per key channel, sigmoid(low-rank projection)^(1 / tau); the head outputs are normed
    with one weight shared by the heads and gated with SiLU."""
    per_head_norm = True

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, slots: int):
        super().__init__(mo.KIND_GLA, w, ["a1"], m["heads"], m["dim"], m["vdim"], eps, dtype, device, slots)
        rank = w["a1"].shape[0]
        a2, a2b = _f32(w["a2"].float().t(), device), _f32(w["a2.b"], device)
        if tuple(w["a2"].shape) != (self.H * self.D, rank):
            raise ValueError(f"a2: shape {tuple(w['a2'].shape)}, expected {(self.H * self.D, rank)}")
        self.keep += [a2, a2b]
        self.desc.update(oa=self.proj.at["a1"], a2=a2.data_ptr(), a2b=a2b.data_ptr(), rank=rank, inv_tau=1.0 / float(m["tau"]))


def rotary_frequencies(dims: int, base: float, scaling: dict | None = None) -> tuple[torch.Tensor, float]:
    """Angular frequency of every rotated pair (float64) and the factor on cos and sin. `scaling` = YaRN's {factor, original,
    fast, slow}: pairs that turn fewer than `slow` times over the original context are slowed down by `factor`, those that
    turn more than `fast` times keep their frequency, with a linear ramp over the pair index between."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / dims)
    if not scaling:
        return f, 1.0
    turn = lambda t: dims * math.log(scaling["original"] / (t * 2.0 * math.pi)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turn(scaling["fast"])), 0), min(math.ceil(turn(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / float(scaling["factor"]) * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


class LatentAttentionMixer:
    """Latent attention over pages of [latent | rotated key part], optional sliding window and sinks. Few rows (decode) score
    queries mapped into the latent space against the cached rows; long portions in bf16 expand the keys and values they can
    see with one GEMM and run the tensor-core kernel."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, pages: int, context: int):
        H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        self.H, self.D, self.R, self.V, self.K, self.eps, self.dtype = H, D, R, V, K, eps, dtype
        self.scale = float(m["scale"])
        self.window = int((m.get("mask") or {}).get("size") or 0)
        for n, shape in (("q", (H * (D + R), None)), ("dkv", (K + R, None)), ("uk", (H * D, K)), ("uv", (H * V, K))):
            if w[n].shape[0] != shape[0] or (shape[1] is not None and w[n].shape[1] != shape[1]):
                raise ValueError(f"{n}: shape {tuple(w[n].shape)}, expected {shape}")
        if m["rot"]["dims"] != R:
            raise ValueError("the rotated dimensions are the rotated part of the head")
        freq, self.mag = rotary_frequencies(R, m["rot"]["base"], m["rot"].get("scaling"))
        self.freq = freq.to(device)
        self.proj = FusedLinear([("q", w["q"]), ("dkv", w["dkv"])], dtype, device)
        self.out = FusedLinear([("o", w["o"])], dtype, device)
        self.c_norm = _f32(w["dkv.norm"], device)
        self.sink = _f32(w["sink"], device) if "sink" in w else None
        self.uk, self.uv = w["uk"].to(dtype).contiguous().to(device), w["uv"].to(dtype).contiguous().to(device)
        self.row = pad_to(K + R, 64)
        self.cache = torch.zeros(pages, mo.PAGE, self.row, dtype=dtype, device=device)
        span = min(self.window, context) if self.window else context
        self.nsplit = max(1, min(64, (span + 31) // 32))
        # expanded keys [k | rotated part] and values as one matrix over a cached row; the rotated part passes through
        self.qk_panels, self.v_panels = pad_to(D + R, 64) // 64, (V + 63) // 64
        if self.v_panels > 1:
            self.v_panels = pad_to(self.v_panels, 2)
        self.tensor_core = dtype == torch.bfloat16 and self.qk_panels <= 4
        self.kv_w = None
        if self.tensor_core:
            qw, vw = self.qk_panels * 64, self.v_panels * 64
            kv = torch.zeros(H * (qw + vw), self.row, dtype=dtype)
            ks, vs = kv[:H * qw].view(H, qw, self.row), kv[H * qw:].view(H, vw, self.row)
            ks[:, :D, :K] = w["uk"].to(dtype).view(H, D, K)
            ks[:, D:D + R, K:K + R] = torch.eye(R, dtype=dtype)
            vs[:, :V, :K] = w["uv"].to(dtype).view(H, V, K)
            self.kv_w = kv.to(device)

    def cache_bytes(self) -> int:
        return self.cache.numel() * self.cache.element_size()

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        T, ws, H, D, R, K, V = ctx.T, ctx.ws, self.H, self.D, self.R, self.K, self.V
        p = self.proj(ctx, h, "proj", torch.float32)
        oq, oc = self.proj.at["q"], self.proj.at["dkv"]
        # rows that attend one by one: those of short portions, or all of them when the tensor-core form does not apply
        long = ctx.n_long > 0 and self.tensor_core
        rows, nrows = (ctx.rows, ctx.n_rows) if long or not ctx.n_long else (ctx.all_rows, T)
        qx = ws.flat("qx", T * H * self.row, torch.float32) if nrows else None
        qw = self.qk_panels * 64
        qf = ws.flat("qf", T * H * qw, torch.bfloat16) if long else None
        mo.latent_prep(p, oq, oc, H, D, R, K, self.c_norm, self.eps, self.freq, self.mag, ctx.pos, ctx.slot, self.cache, ctx.table, qx, qf, qw)
        mix = ws.rows("mix", T, self.out.K, self.dtype)
        if long:
            gather, total, longest = ctx.gather[self.window]
            c = ws.rows("lat_rows", total, self.row, torch.bfloat16)
            mo.latent_gather(self.cache, ctx.table, ctx.long, gather, ctx.n_long, longest, c)
            kv = ws.rows("lat_kv", total, self.kv_w.shape[0], torch.bfloat16)
            mo.linear(c, self.kv_w, kv, ctx.status)
            mo.latent_prefill(qf, T, kv, total, ctx.tiles, ctx.n_tiles, ctx.long, gather, H, self.qk_panels, self.v_panels, V, self.window, self.scale,
                              self.sink, mix, ctx.status)
        if nrows:
            mo.latent_absorb(p, oq, H, D, R, K, self.uk, rows, nrows, qx, self.row)
            per = max(8, (64 << 20) // (self.nsplit * H * K))
            for a in range(0, nrows, per):
                n = min(per, nrows - a)
                po, pm = ws.flat("part_o", n * self.nsplit * H * K, torch.float32), ws.flat("part_ml", n * self.nsplit * H * 2, torch.float32)
                r = rows[a:a + n]
                mo.latent_rows(qx, r, n, ctx.pos, ctx.slot, self.cache, ctx.table, H, K, self.window, self.scale, self.nsplit, po, pm)
                mo.latent_out(po, pm, self.nsplit, H, K, V, self.sink, r, n, self.uv, mix)
        return self.out(ctx, mix, "y", torch.float32)


class SwiGLU:
    """W_down (silu(W_gate h) * (W_up h)); the hidden size is padded to what the GEMM's epilogue takes."""

    def __init__(self, w: dict, dtype, device):
        ff, K = w["gate"].shape
        self.ff, self.dtype = pad_to(ff, 128), dtype
        gu = torch.zeros(2 * self.ff, pad_to(K, 64), dtype=dtype)
        gu[:ff, :K], gu[self.ff:self.ff + ff, :K] = w["gate"].to(dtype), w["up"].to(dtype)
        self.gate_up = gu.to(device)
        self.down = FusedLinear([("down", w["down"])], dtype, device, k_pad=self.ff)

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        mid = ctx.ws.rows("mid", ctx.T, self.ff, self.dtype)
        mo.linear(h, self.gate_up, mid, ctx.status, swiglu=True)
        return self.down(ctx, mid, "y", torch.float32)


@dataclass
class SandwichLayer:
    """A mixer and an optional feed-forward, each between two norms."""
    mixer: object
    norm1: torch.Tensor
    norm1b: torch.Tensor
    mlp: SwiGLU | None = None
    norm2: torch.Tensor | None = None
    norm2b: torch.Tensor | None = None


@dataclass
class MixerModel:
    """What `runtime.mixer_runtime.MixerRuntime` runs: an embedding, layers, a final norm and an output matrix."""
    vocab: int
    width: int
    eps: float
    dtype: torch.dtype
    embed: torch.Tensor            # [vocab, width] bf16
    layers: list[SandwichLayer]
    final_norm: torch.Tensor
    head: FusedLinear
    plus_one: bool = True          # norm weights are stored around zero

    def windows(self) -> set[int]:
        return {L.mixer.window for L in self.layers if isinstance(L.mixer, LatentAttentionMixer)}


MIXERS = {"mlstm": MLSTMMixer, "gla": GLAMixer, "latent_attention": LatentAttentionMixer}
PAGED = {"latent_attention"}
