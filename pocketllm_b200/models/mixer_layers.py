"""Layers of decoders that are put together from mixers: every layer names its kind of mixer (recurrent state or attention)
and optionally a feed-forward, with its own sizes. The classes here hold a layer's weights in the layout of the kernels,
the device memory of its state or cache, and its forward pass over a mixed batch (`StepContext`): portions of prompts
beside single decoded tokens, any request in any slot.

Two precisions: bfloat16 (bf16 weights, activations and cache, fp32 accumulation; norms, gates, recurrences, attention
scores and the residual stream in fp32) and float32 (everything, without reduced-precision tensor modes).
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field, replace

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
    behind: torch.Tensor                 # tokens of the same portion after a row
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
    tile0: torch.Tensor | None = None   # first tile of every long portion
    gather: dict = field(default_factory=dict)   # window -> ({first key row, its position} per long sequence, key rows, longest)


class FusedLinear:
    """Row blocks of several matrices that share their input as one [N, K] matrix, padded with zeros to what the kernels
    take; `at[name]` is the first output column of a block (a multiple of `align`). The blocks of `beside` come first and have an
    input of their own."""

    def __init__(self, blocks: list[tuple[str, torch.Tensor]], dtype: torch.dtype, device, k_pad: int | None = None, align: int = 1,
                 beside: list[tuple[str, torch.Tensor]] | None = None):
        K = blocks[0][1].shape[1]
        self.K = k_pad or pad_to(K, 64)
        self.at, n = {}, 0
        self.split = 0
        for part in (beside or [], blocks):
            self.split = n = pad_to(n, 8)
            for name, w in part:
                if w.shape[1] != K:
                    raise ValueError(f"{name}: {w.shape[1]} input columns, the others have {K}")
                self.at[name] = n = pad_to(n, align)
                n += w.shape[0]
        self.N = pad_to(n, 8)
        w = torch.zeros(self.N, self.K, dtype=dtype)
        for name, b in (beside or []) + blocks:
            w[self.at[name]:self.at[name] + b.shape[0], :K] = b.to(dtype)
        self.w = w.to(device)

    def __call__(self, ctx: StepContext, x: torch.Tensor, name: str, dtype: torch.dtype, beside: torch.Tensor | None = None) -> torch.Tensor:
        out = ctx.ws.rows(name, x.shape[0], self.N, dtype)
        if self.split:
            return mo.linear2(beside, x, self.split, self.w, out, ctx.status)
        return mo.linear(x, self.w, out, ctx.status)


def _f32(t: torch.Tensor, device) -> torch.Tensor:
    return t.float().contiguous().to(device)


class RecurrentMixer:
    """Base of the mixers with an outer-product state per head. Subclasses fill `self.desc` with what is theirs. `beside`: matrices
    that the projection carries along for its owner (see `FusedLinear`)."""
    per_head_norm = False
    inputs = ("q", "k", "v", "g")

    def __init__(self, kind: int, w: dict, extra: list[str], heads: int, dim: int, vdim: int, eps: float, dtype, device, slots: int, beside=None):
        if dim > 512:
            raise ValueError("recurrent mixers take key dims up to 512")
        self.H, self.D, self.V, self.eps, self.dtype = heads, dim, vdim, eps, dtype
        for n, r in (("q", heads * dim), ("k", heads * dim), ("f", heads * dim), ("v", heads * vdim), ("g", heads * vdim)):
            if n in self.inputs and w[n].shape[0] != r:
                raise ValueError(f"{n}: {w[n].shape[0]} rows, expected {r}")
        self.proj = FusedLinear([(n, w[n]) for n in [*self.inputs, *extra]], dtype, device, beside=beside)
        self.out = FusedLinear([("o", w["o"])], dtype, device)
        self.norm = _f32(w["norm"], device) if "norm" in w else None
        self.S = torch.zeros(slots, heads, dim, vdim, device=device)
        self.N = self.Ms = None
        a = self.proj.at
        self.keep: list[torch.Tensor] = []
        self.desc = dict(kind=kind, H=heads, D=dim, V=vdim, qscale=dim ** -0.5, S=self.S.data_ptr(), **{"o" + n: a[n] for n in self.inputs})

    def again(self):
        """The same weights with states of their own (a further pass over the layer)."""
        o = copy.copy(self)
        o.desc = dict(self.desc)
        for n in ("S", "N", "Ms"):
            t = getattr(self, n)
            if t is not None:
                setattr(o, n, torch.zeros_like(t))
                o.desc[n] = getattr(o, n).data_ptr()
        return o

    def state_bytes(self) -> int:
        return sum(t.numel() * 4 for t in (self.S, self.N, self.Ms) if t is not None)

    def forward(self, ctx: StepContext, h: torch.Tensor, beside: torch.Tensor | None = None) -> torch.Tensor:
        T, ws = ctx.T, ctx.ws
        p = self.proj(ctx, h, "proj", torch.float32, beside)
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


class RetentionMixer(RecurrentMixer):
    """Linear attention with a constant decay per head and rotary positions; the head outputs are normed without a weight and
    gated with SiLU."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, slots: int):
        super().__init__(mo.KIND_RETENTION, w, [], m["heads"], m["dim"], m["vdim"], eps, dtype, device, slots)
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        freq = rotary_frequencies(rot["dims"], rot["base"])[0].to(device)
        decay = torch.tensor([float(a) for a in m["decay"]], dtype=torch.float64)
        powers = (decay[:, None] ** torch.arange(mo.CHUNK + 1, dtype=torch.float64)).float().to(device)
        self.keep += [freq, powers]
        self.desc.update(freq=freq.data_ptr() if rot["dims"] else None, rot=rot["dims"], pw=powers.data_ptr())


class HGRN2Mixer(RecurrentMixer):
    """Linear attention whose forget gate is also its key: a channel keeps f and is written with 1 - f, f = l + (1 - l) sigmoid(.) above
    a lower bound l; queries pass SiLU; the head outputs are normed with one weight shared by the heads."""
    per_head_norm = True
    inputs = ("q", "f", "v")

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, slots: int, beside=None):
        super().__init__(mo.KIND_HGRN, w, [], m["heads"], m["dim"], m["vdim"], eps, dtype, device, slots, beside)
        bias, low = _f32(w["f.b"], device), _f32(w["lower"], device)
        self.keep += [bias, low]
        self.desc.update(qscale=1.0, bf=bias.data_ptr(), low=low.data_ptr())


class SelectiveScanMixer:
    """The selective scan of Mamba: x through a short convolution, step sizes (from a low-rank projection), B and C from x, a decay per
    channel and state, SiLU gate."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, slots: int, beside=None):
        inner, N, rank, taps = m["inner"], m["state"], m["dt_rank"], m["conv"]
        self.inner, self.N, self.rank, self.taps, self.dtype = inner, N, rank, taps, dtype
        if N > 256:
            raise ValueError("selective scans take states up to 256")
        for n, s in (("in", (2 * inner, None)), ("conv", (inner, taps)), ("conv.b", (inner,)), ("x", (rank + 2 * N, inner)), ("dt", (inner, rank)),
                     ("dt.b", (inner,)), ("A_log", (inner, N)), ("D", (inner,)), ("o", (None, inner))):
            if any(b is not None and a != b for a, b in zip(w[n].shape, s)):
                raise ValueError(f"{n}: shape {tuple(w[n].shape)}, expected {s}")
        self.proj = FusedLinear([("x", w["in"][:inner]), ("z", w["in"][inner:])], dtype, device, align=4, beside=beside)
        self.dbc = FusedLinear([("d", w["x"][:rank]), ("B", w["x"][rank:rank + N]), ("C", w["x"][rank + N:])], dtype, device, align=4)
        self.out = FusedLinear([("o", w["o"])], dtype, device)
        # step sizes: few rows read the plain matrix, many rows multiply it with a two-term input in bf16
        kw = pad_to(rank, 32)
        wide = torch.zeros(inner, kw if dtype == torch.float32 else 2 * kw)
        for a in range(0, wide.shape[1], kw):
            wide[:, a:a + rank] = w["dt"]
        self.dt = FusedLinear([("dt", wide)], dtype, device, k_pad=wide.shape[1])
        self.kw = kw
        f = lambda n: _f32(w[n], device)
        decay = (-torch.exp(w["A_log"].double()) * (math.log2(math.e) if dtype == torch.bfloat16 else 1.0)).float().contiguous().to(device)
        self.const = {"cw": f("conv"), "cb": f("conv.b"), "dt_bias": f("dt.b"), "A": decay, "skip": f("D"), "w_dt": self.dt.w}
        self.desc = dict(ox=self.proj.at["x"], oz=self.proj.at["z"], oB=self.dbc.at["B"], oC=self.dbc.at["C"], ldw=self.dt.K, inner=inner, N=N, rank=rank, taps=taps, f32=int(dtype == torch.float32),
                         **{n: t.data_ptr() for n, t in self.const.items()})
        self._memory(slots, device)

    def _memory(self, slots: int, device) -> None:
        self.S = torch.zeros(slots, self.inner, self.N, device=device)
        self.ring = torch.zeros(slots, max(self.taps - 1, 1), self.inner, device=device)
        self.desc = dict(self.desc, S=self.S.data_ptr(), ring=self.ring.data_ptr())

    def again(self):
        """The same weights with states of their own."""
        o = copy.copy(self)
        o._memory(self.S.shape[0], self.S.device)
        return o

    def state_bytes(self) -> int:
        return (self.S.numel() + self.ring.numel()) * 4

    def forward(self, ctx: StepContext, h: torch.Tensor, beside: torch.Tensor | None = None) -> torch.Tensor:
        p = self.proj(ctx, h, "proj", torch.float32, beside)
        mix = ctx.ws.rows("mix", ctx.T, self.out.K, self.dtype)
        self.run(ctx, p, mix)
        return self.out(ctx, mix, "y", torch.float32)

    def run(self, ctx: StepContext, p: torch.Tensor, mix: torch.Tensor) -> None:
        T, ws = ctx.T, ctx.ws
        x = ws.rows("scan_x", T, self.dbc.K, self.dtype)
        d = mo.SelectiveScan(proj=p.data_ptr(), ld=p.stride(0), xc=x.data_ptr(), ldx=x.stride(0), out=mix.data_ptr(), ldo=mix.stride(0),
                             pos=ctx.pos.data_ptr(), slot=ctx.slot.data_ptr(), **self.desc)
        mo.scan_conv(d, T)
        dbc = self.dbc(ctx, x, "scan_dbc", torch.float32)
        d.dbc, d.ldb = dbc.data_ptr(), dbc.stride(0)
        if ctx.n_short:
            mo.scan_rows(d, ctx.short, ctx.n_short)
        if ctx.n_long:
            terms = ws.rows("scan_d", T, self.dt.K, self.dtype)
            if self.dtype == torch.bfloat16:
                mo.scan_split(dbc, self.rank, terms)
            else:
                terms[:, self.rank:] = 0
                terms[:, :self.rank] = dbc[:, :self.rank]
            dt = self.dt(ctx, terms, "scan_dt", torch.float32)
            d.dt, d.ldt = dt.data_ptr(), dt.stride(0)
            mo.scan_tiles(d, ctx.long, ctx.n_long)


class StateSpaceMixer:
    """The state-space recurrence of Mamba-2: x, B and C through a short convolution, a scalar decay per token and head, gate before
    a norm in equal parts. `scale` multiplies its output. Works on columns of a projection that its owner makes. Long portions in
    bf16 run on the tensor cores where the shape fits them."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, slots: int, scale: float = 1.0):
        H, V, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
        self.H, self.V, self.N, self.parts, self.eps, self.dtype = H, V, N, m["norm_groups"], eps, dtype
        if N > 512:
            raise ValueError("state-space layers take states up to 512")
        ch = H * V + 2 * G * N
        for n, s in (("in", (2 * H * V + 2 * G * N + H, None)), ("conv", (ch, taps)), ("conv.b", (ch,)), ("dt_bias", (H,)), ("A_log", (H,)), ("D", (H,)),
                     ("norm", (H * V,))):
            if any(b is not None and a != b for a, b in zip(w[n].shape, s)):
                raise ValueError(f"{n}: shape {tuple(w[n].shape)}, expected {s}")
        f = lambda n: _f32(w[n], device)
        self.const = {"cw": f("conv"), "cb": f("conv.b"), "dtb": f("dt_bias"), "A": -torch.exp(w["A_log"].double()).float().to(device), "skip": f("D")}
        self.norm = f("norm") * scale
        self.S = torch.zeros(slots, H, N, V, device=device)
        self.ring = torch.zeros(slots, max(taps - 1, 1), ch, device=device)
        self.desc = dict(kind=mo.KIND_SSD, H=H, D=N, V=V, groups=G, taps=taps, qscale=1.0, S=self.S.data_ptr(), Cs=self.ring.data_ptr(),
                         **{n: t.data_ptr() for n, t in self.const.items()})

    def at(self, first: int) -> None:
        """The projection's columns z | x B C | dt start at `first`."""
        inner = self.H * self.V
        self.desc.update(og=first, ov=first + inner, odt=first + 2 * inner + 2 * self.desc["groups"] * self.N)

    def state_bytes(self) -> int:
        return (self.S.numel() + self.ring.numel()) * 4

    def run(self, ctx: StepContext, p: torch.Tensor, out: torch.Tensor) -> None:
        ws = ctx.ws
        o = ws.flat("raw_o", ctx.T * self.H * self.V, torch.float32)
        d = mo.StateMixer(proj=p.data_ptr(), ld=p.stride(0), o=o.data_ptr(), **self.desc)
        if ctx.n_short:
            mo.ssd_rows(d, ctx.short, ctx.n_short)
        if ctx.n_long:
            n = mo.ssd_tile_workspace(d, ctx.n_tiles) if self.dtype == torch.bfloat16 else 0
            if n:
                mo.ssd_tiles(d, ctx.long, ctx.n_long, ctx.tiles, ctx.tile0, ctx.n_tiles, ws.flat("state_chunks", n, torch.float32), ctx.status)
            else:
                scratch = ws.flat("state_chunks", mo.state_chunk_workspace(d, ctx.n_chunks), torch.float32)
                mo.state_chunks(d, ctx.long, ctx.n_long, ctx.chunks, ctx.chunk0, ctx.n_chunks, scratch)
        mo.ssd_out(d, self.norm, self.parts, self.eps, ctx.slot, ctx.behind, ctx.pos, ctx.T, out)


def rotary_frequencies(dims: int, base: float, scaling: dict | None = None) -> tuple[torch.Tensor, float]:
    """Angular frequency of every rotated pair (float64) and the factor on cos and sin. `scaling` = {factor} slows every pair down
    alike; YaRN's {factor, original, fast, slow}: pairs that turn fewer than `slow` times over the original context are slowed down
    by `factor`, those that turn more than `fast` times keep their frequency, with a linear ramp over the pair index between."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / max(dims, 1))
    if not scaling:
        return f, 1.0
    if "original" not in scaling:
        return f / float(scaling["factor"]), 1.0
    turn = lambda t: dims * math.log(scaling["original"] / (t * 2.0 * math.pi)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turn(scaling["fast"])), 0), min(math.ceil(turn(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / float(scaling["factor"]) * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


class LatentAttentionMixer:
    """Latent attention over pages of [latent | rotated key part], optional sliding window and sinks. Few rows (decode) score
    queries mapped into the latent space against the cached rows; long portions in bf16 expand the keys and values they can
    see with one GEMM and run the tensor-core kernel. Without a rotated part (`rot_dim` missing) the queries may come from a latent of
    their own (`dq`, `dq.norm`, `uq` among the weights instead of `q`); `g` among the weights: a sigmoid gate on the heads' outputs."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, pages: int, context: int, beside=None):
        H, D, R, V, K = m["heads"], m["dim"], m.get("rot_dim") or 0, m["vdim"], m["kv_rank"]
        self.q_rank = w["dq"].shape[0] if "dq" in w else 0
        self.H, self.D, self.R, self.V, self.K, self.eps, self.dtype = H, D, R, V, K, eps, dtype
        self.scale = float(m["scale"])
        self.window = int((m.get("mask") or {}).get("size") or 0)
        for n, shape in (("q", (H * (D + R), None)), ("uq", (H * D, self.q_rank)), ("dkv", (K + R, None)), ("uk", (H * D, K)), ("uv", (H * V, K)), ("g", (H * V, None))):
            if n in w and (w[n].shape[0] != shape[0] or (shape[1] is not None and w[n].shape[1] != shape[1])):
                raise ValueError(f"{n}: shape {tuple(w[n].shape)}, expected {shape}")
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        if rot["dims"] != R or (R and self.q_rank):
            raise ValueError("the rotated dimensions are the rotated part of the head; queries from a latent have none")
        freq, self.mag = rotary_frequencies(R, rot["base"], rot.get("scaling"))
        self.freq = freq.to(device)
        self.proj = FusedLinear([(n, w[n]) for n in ("q", "dq", "dkv", "g") if n in w], dtype, device, align=4, beside=beside)
        self.gated = "g" in w
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
        if self.q_rank:      # heads of the expanded queries start where the tensor-core kernel wants them
            uq = torch.zeros(H, self.qk_panels * 64, self.q_rank, dtype=dtype)
            uq[:, :D] = w["uq"].to(dtype).view(H, D, self.q_rank)
            self.uq = FusedLinear([("q", uq.view(-1, self.q_rank))], dtype, device)
            self.q_norm = _f32(w["dq.norm"], device)
        self.kv_w = None
        if self.tensor_core:
            qw, vw = self.qk_panels * 64, self.v_panels * 64
            kv = torch.zeros(H * (qw + vw), self.row, dtype=dtype)
            ks, vs = kv[:H * qw].view(H, qw, self.row), kv[H * qw:].view(H, vw, self.row)
            ks[:, :D, :K] = w["uk"].to(dtype).view(H, D, K)
            ks[:, D:D + R, K:K + R] = torch.eye(R, dtype=dtype)
            vs[:, :V, :K] = w["uv"].to(dtype).view(H, V, K)
            self.kv_w = kv.to(device)

    def again(self):
        o = copy.copy(self)
        o.cache = torch.zeros_like(self.cache)
        return o

    def cache_bytes(self) -> int:
        return self.cache.numel() * self.cache.element_size()

    def forward(self, ctx: StepContext, h: torch.Tensor, beside: torch.Tensor | None = None) -> torch.Tensor:
        T, ws, H, D, R, K, V = ctx.T, ctx.ws, self.H, self.D, self.R, self.K, self.V
        p = self.proj(ctx, h, "proj", torch.float32, beside)
        at = self.proj.at
        gate = p[:, at["g"]:] if self.gated else None
        # rows that attend one by one: those of short portions, or all of them when the tensor-core form does not apply
        long = ctx.n_long > 0 and self.tensor_core
        rows, nrows = (ctx.rows, ctx.n_rows) if long or not ctx.n_long else (ctx.all_rows, T)
        qx = ws.flat("qx", T * H * self.row, torch.float32) if nrows else None
        qw = self.qk_panels * 64
        if self.q_rank:
            ql = ws.rows("lat_q", T, self.uq.K, self.dtype)
            mo.latent_prep(p, at["dq"], at["dkv"], H, D, R, K, self.c_norm, self.eps, self.freq, self.mag, ctx.pos, ctx.slot, self.cache, ctx.table, None, None, 0,
                           q_rank=self.q_rank, q_norm=self.q_norm, ql=ql)
            qf = self.uq(ctx, ql, "qf", torch.bfloat16) if long else None
            q, oq, gap, k_pad = (self.uq(ctx, ql, "q_rows", torch.float32) if nrows else None), 0, qw - D, self.row
        else:
            qf = ws.flat("qf", T * H * qw, torch.bfloat16) if long else None
            mo.latent_prep(p, at["q"], at["dkv"], H, D, R, K, self.c_norm, self.eps, self.freq, self.mag, ctx.pos, ctx.slot, self.cache, ctx.table, qx, qf, qw)
            q, oq, gap, k_pad = p, at["q"], R, K
        mix = ws.rows("mix", T, self.out.K, self.dtype)
        if long:
            gather, total, longest = ctx.gather[self.window]
            c = ws.rows("lat_rows", total, self.row, torch.bfloat16)
            mo.latent_gather(self.cache, ctx.table, ctx.long, gather, ctx.n_long, longest, c)
            kv = ws.rows("lat_kv", total, self.kv_w.shape[0], torch.bfloat16)
            mo.linear(c, self.kv_w, kv, ctx.status)
            mo.latent_prefill(qf, T, kv, total, ctx.tiles, ctx.n_tiles, ctx.long, gather, H, self.qk_panels, self.v_panels, V, self.window, self.scale,
                              self.sink, mix, ctx.status, gate)
        if nrows:
            mo.latent_absorb(q, oq, H, D, gap, K, self.uk, rows, nrows, qx, self.row, k_pad)
            per = max(8, (64 << 20) // (self.nsplit * H * K))
            for a in range(0, nrows, per):
                n = min(per, nrows - a)
                po, pm = ws.flat("part_o", n * self.nsplit * H * K, torch.float32), ws.flat("part_ml", n * self.nsplit * H * 2, torch.float32)
                r = rows[a:a + n]
                mo.latent_rows(qx, r, n, ctx.pos, ctx.slot, self.cache, ctx.table, H, K, self.window, self.scale, self.nsplit, po, pm)
                mo.latent_out(po, pm, self.nsplit, H, K, V, self.sink, r, n, self.uv, mix, gate)
        return self.out(ctx, mix, "y", torch.float32)


class GroupedAttention:
    """Grouped-query attention over pages of [keys | values]: causal, in a window or in chunks (`mask`), rotary positions on a
    leading part of every query and key. Works on columns of a projection that its owner makes. Options of a design:
      * `q.norm`, `k.norm` among the weights: norms of queries and keys before the rotation
      * `neighbours`: rotated pairs are (2i, 2i + 1) instead of half a width apart
      * `softcap` in the configuration: scores become cap tanh(score / cap)
      * `sink`: score of a key without a value that every query sees
      * `g` among the weights: a sigmoid gate per head on its output
      * `v_mix` = "first" | "mix": the values are kept for later layers, or become (1 - vmix) v + vmix x (the kept ones)
      * `diff` in the configuration: a head has two softmax maps over the same values, its output is a1 - lambda a2, normed without
        a weight and scaled by 1 - diff
      * `scale_out`: a factor on the outputs
    Long portions in bf16 run the tensor-core kernel on the pages, everything else the row kernel."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, pages: int, context: int, mask: str = "window", neighbours: bool = False,
                 sink: float | None = None, v_mix: str | None = None, scale_out: float = 1.0):
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        diff = m.get("diff")
        maps = 1 if diff is None else 2
        if V > 512:
            raise ValueError("attention takes value dims up to 512")
        for n, r in (("q", H * maps * D), ("k", G * maps * D), ("v", G * V), ("g", H), ("q.norm", D), ("k.norm", D)):
            if n in w and w[n].shape[0] != r:
                raise ValueError(f"{n}: {w[n].shape[0]} rows, expected {r}")
        self.H, self.G, self.D, self.V, self.maps, self.dtype = H, G, D, V, maps, dtype
        size = int((m.get("mask") or {}).get("size") or 0)
        self.span = min(size, context) if size else context         # most positions a query sees
        self.nsplit = max(1, min(64, (self.span + 31) // 32))
        dp, vp = pad_to(D, 8), pad_to(V, 8)
        self.row = G * (maps * dp + vp)
        self.q_ld = pad_to(D, 64)
        self.tensor_core = dtype == torch.bfloat16 and float(m["scale"]) > 0
        self.cache = torch.zeros(pages, mo.PAGE, self.row, dtype=dtype, device=device)
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        freq, mag = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        if mag != 1.0:
            raise ValueError("grouped attention does not scale its rotations")
        self.const = {"freq": freq.to(device)}                     # keeps what the descriptor points at
        self.desc = dict(H=H, G=G, maps=maps, D=D, V=V, R=rot["dims"], dp=dp, vp=vp, row=self.row, f32=int(dtype == torch.float32),
                         window=size if mask == "window" else 0, chunk=size if mask == "chunk" else 0, q_ld=self.q_ld, scale=float(m["scale"]), eps=eps,
                         post=scale_out, neighbours=int(neighbours), gate=-1, cap=float(m.get("softcap") or 0.0), cache=self.cache.data_ptr())
        for n, key in (("q.norm", "q_norm"), ("k.norm", "k_norm")):
            if n in w:
                self.const[key] = _f32(w[n], device)
        if sink is not None:
            self.const["sink"] = torch.full((H * maps,), float(sink), device=device)
        self.desc.update({n: t.data_ptr() if t.numel() else None for n, t in self.const.items()})
        if v_mix:
            self.desc["v_mix"] = {"first": 1, "mix": 2}[v_mix]
            if v_mix == "mix":
                self.desc["mix"] = float(w["vmix"])
        if maps == 2:
            l = {n: w[n].double() for n in ("lq1", "lk1", "lq2", "lk2")}
            lam = float(torch.exp((l["lq1"] * l["lk1"]).sum()) - torch.exp((l["lq2"] * l["lk2"]).sum())) + float(diff)
            self.desc.update(lambda_=lam, head_norm=1, post=scale_out * (1.0 - float(diff)))

    @staticmethod
    def blocks(w: dict) -> list[tuple[str, torch.Tensor]]:
        """Matrices of the projection."""
        return [(n, w[n]) for n in ("q", "k", "v", "g") if n in w]

    def at(self, columns: dict, prefix: str = "") -> None:
        """Where the blocks of the projection start."""
        self.desc.update({k: columns[prefix + n] for n, k in (("q", "oq"), ("k", "ok"), ("v", "ov"), ("g", "gate")) if prefix + n in columns})

    def own_memory(self) -> None:
        self.cache = torch.zeros_like(self.cache)
        self.desc = dict(self.desc, cache=self.cache.data_ptr())

    def cache_bytes(self) -> int:
        return self.cache.numel() * self.cache.element_size()

    def describe(self, ctx: StepContext, p: torch.Tensor, out: torch.Tensor) -> mo.PagedAttention:
        d = mo.PagedAttention(proj=p.data_ptr(), ld=p.stride(0), pos=ctx.pos.data_ptr(), slot=ctx.slot.data_ptr(), table=ctx.table.data_ptr(),
                              table_ld=ctx.table.stride(0), out=out.data_ptr(), ldo=out.stride(0), width=out.shape[1], status=ctx.status.data_ptr(),
                              nsplit=1, **self.desc)
        if d.v_mix:
            d.v_first = ctx.ws.flat("v_first", ctx.T * self.G * self.V, torch.float32).data_ptr()
        return d

    def run(self, ctx: StepContext, p: torch.Tensor, out: torch.Tensor) -> None:
        """Head outputs of all rows into `out` [rows, columns of this layer] (a view is fine)."""
        T, ws, nq = ctx.T, ctx.ws, self.H * self.maps
        d = self.describe(ctx, p, out)
        form = mo.paged_prefill_form(self.maps, self.D, self.V) if ctx.n_long and self.tensor_core else -1
        rows, nrows = (ctx.rows, ctx.n_rows) if form >= 0 or not ctx.n_long else (ctx.all_rows, T)
        if nrows:
            d.qx = ws.flat("qx", T * nq * self.D, torch.float32).data_ptr()
        if form >= 0:
            d.qf = ws.flat("qf", T * nq * self.q_ld, torch.bfloat16).data_ptr()
        mo.paged_prep(d, T)
        if form >= 0:
            if form == 0:
                d.part_o = ws.flat("raw_o", T * nq * self.V, torch.float32).data_ptr()
            mo.paged_prefill(d, T, self.cache.shape[0], ctx.tiles, ctx.n_tiles, ctx.long)
            if form == 0:
                mo.paged_merge(d, None, T)         # rows of short portions are written again below
        if nrows:
            d.nsplit = self.nsplit if nrows <= 64 else 1
            per = max(8, (64 << 20) // (d.nsplit * nq * self.V))
            for a in range(0, nrows, per):
                n = min(per, nrows - a)
                d.part_o = ws.flat("part_o", n * d.nsplit * nq * self.V, torch.float32).data_ptr()
                d.part_ml = ws.flat("part_ml", n * d.nsplit * nq * 2, torch.float32).data_ptr()
                mo.paged_rows(d, rows[a:a + n], n)
                mo.paged_merge(d, rows[a:a + n], n)


class GroupedAttentionMixer(GroupedAttention):
    """Grouped-query attention between a projection and an output matrix of its own."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, pages: int, context: int, **options):
        super().__init__(w, m, eps, dtype, device, pages, context, **options)
        self.proj = FusedLinear(self.blocks(w), dtype, device)
        self.out = FusedLinear([("o", w["o"])], dtype, device)
        self.at(self.proj.at)

    def again(self):
        o = copy.copy(self)
        o.own_memory()
        return o

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        p = self.proj(ctx, h, "proj", torch.float32)
        mix = ctx.ws.rows("mix", ctx.T, self.out.K, self.dtype)
        self.run(ctx, p, mix)
        return self.out(ctx, mix, "y", torch.float32)


class ParallelMixer:
    """Attention and a state-space recurrence side by side on the same input: one projection in front of both and one output matrix
    behind both, their outputs laid end to end. What scales a side is part of its last factor (attention) or its norm's weight."""

    def __init__(self, left: GroupedAttention, right: StateSpaceMixer, w_left: dict, w_right: dict, dtype, device):
        self.left, self.right, self.dtype = left, right, dtype
        self.proj = FusedLinear([("left." + n, t) for n, t in left.blocks(w_left)] + [("right", w_right["in"])], dtype, device, align=4)
        left.at(self.proj.at, "left.")
        right.at(self.proj.at["right"])
        n = left.H * left.V
        self.split = pad_to(n, 8)
        o = torch.zeros(w_left["o"].shape[0], self.split + right.H * right.V, dtype=w_left["o"].dtype)
        o[:, :n], o[:, self.split:] = w_left["o"], w_right["o"]
        self.out = FusedLinear([("o", o)], dtype, device)

    def cache_bytes(self) -> int:
        return self.left.cache_bytes()

    def state_bytes(self) -> int:
        return self.right.state_bytes()

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        p = self.proj(ctx, h, "proj", torch.float32)
        mix = ctx.ws.rows("mix", ctx.T, self.out.K, self.dtype)
        self.left.run(ctx, p, mix[:, :self.split])
        self.right.run(ctx, p, mix[:, self.split:])
        return self.out(ctx, mix, "y", torch.float32)


class SwiGLU:
    """W_down (silu(W_gate h) * (W_up h)); the hidden size is padded to what the GEMM's epilogue takes. `name`: of its scratch."""

    def __init__(self, w: dict, dtype, device, name: str = ""):
        ff, K = w["gate"].shape
        self.name = name
        self.ff, self.dtype = pad_to(ff, 128), dtype
        gu = torch.zeros(2 * self.ff, pad_to(K, 64), dtype=dtype)
        gu[:ff, :K], gu[self.ff:self.ff + ff, :K] = w["gate"].to(dtype), w["up"].to(dtype)
        self.gate_up = gu.to(device)
        self.down = FusedLinear([("down", w["down"])], dtype, device, k_pad=self.ff)

    def forward(self, ctx: StepContext, h: torch.Tensor) -> dict:
        mid = ctx.ws.rows("mid" + self.name, ctx.T, self.ff, self.dtype)
        mo.linear(h, self.gate_up, mid, ctx.status, swiglu=True)
        return {"y": self.down(ctx, mid, "y" + self.name, torch.float32)}


class RoutedExperts:
    """Routed experts W_down max(W_up x, 0)^2, or with `gate` matrices W_down (silu(W_gate x) * (W_up x)). Few rows (and fp32) stream
    the chosen experts' weights; many rows are grouped by expert and multiplied on the tensor cores, and the sum over a token's
    experts is left to the norm that follows, as is what experts that return their input and a `shared` expert add: `forward` returns
    what `sandwich_norm` or the step of a `PostSum` model takes. `out_gate`: the matrix of a gate on the result, whose logits come with the
    router's."""

    def __init__(self, router_w: torch.Tensor, up: list[torch.Tensor], down: list[torch.Tensor], router: mo.Router, dtype, device,
                 gate: list[torch.Tensor] | None = None, correction: torch.Tensor | None = None, bias: torch.Tensor | None = None,
                 shared: "SwiGLU | None" = None, out_gate: torch.Tensor | None = None):
        E, (ff, K), W = router.experts, up[0].shape, down[0].shape[0]
        self.route, self.W, self.dtype, self.gated = router, W, dtype, gate is not None
        self.router = FusedLinear([("router", router_w)] + ([] if out_gate is None else [("gate", out_gate)]), dtype, device, align=4)
        self.correction, self.bias = (None if t is None else _f32(t, device) for t in (correction, bias))
        self.shared, self.gate_at = shared, self.router.at.get("gate")
        self.ff, kp = pad_to(ff, 128), pad_to(K, 64)
        self.up = torch.zeros(E, self.ff * (2 if gate else 1), kp, dtype=dtype, device=device)
        self.down = torch.zeros(E, pad_to(W, 128), self.ff, dtype=dtype, device=device)
        for e in range(E):
            self.up[e, -self.ff:][:ff, :K] = up[e].to(device=device, dtype=dtype)
            if gate:
                self.up[e, :ff, :K] = gate[e].to(device=device, dtype=dtype)
            self.down[e, :W, :ff] = down[e].to(device=device, dtype=dtype)

    def forward(self, ctx: StepContext, h: torch.Tensor) -> dict:
        T, ws, r = ctx.T, ctx.ws, self.route
        R = T * r.top
        z = self.router(ctx, h, "router", torch.float32)
        ids = ws.flat("route_ids", R, torch.int32)
        hidden = ws.rows("mid", R, self.ff, self.dtype)
        skip_w = ws.flat("route_skip", T, torch.float32) if r.identity else None
        rest = {"skip": h, "skip_w": skip_w} if r.identity else {}
        kw = {"correction": self.correction, "skip_w": skip_w, "bias": self.bias}
        if self.gate_at is not None:
            rest["gate"] = z[:, self.gate_at:]
        if self.shared is not None:
            rest["y2"] = self.shared.forward(ctx, h)["y"]
        if T <= mo.ROWS_MAX or self.dtype == torch.float32:
            mo.expert_up_rows(r, z, h, self.up, ids, hidden, gated=self.gated, **kw)
            y = ws.rows("y", T, self.down.shape[1], torch.float32)
            mo.expert_down_rows(r, ids, hidden, self.down, self.W, y)
            return {"y": y, **rest}
        place = ws.rows("route_place", T, r.top, torch.int32)
        seg, scale = ws.flat("route_seg", r.experts + 1, torch.int32), ws.flat("route_scale", R, torch.float32)
        x = ws.rows("route_x", R, self.up.shape[2], self.dtype)
        mo.expert_group(r, z, h, ids, ws.flat("route_w", R, torch.float32), seg, place, scale, x, **kw)
        mo.grouped_linear(x, self.up, seg, hidden, ctx.status, relu2=not self.gated, swiglu=self.gated, row_scale=scale, scale_after=r.on_output)
        y = ws.rows("expert_y", R, self.down.shape[1], torch.float32)
        mo.grouped_linear(hidden, self.down, seg, y, ctx.status)
        return {"y": y, "y_rows": place, **rest}


@dataclass
class MixerLayer:
    """A mixer and an optional feed-forward, normed before and optionally (`norm1b`, `norm2b`) after; in a `PostSum` model `norm1` and
    `norm2` follow the sums, the mixer may read a mix of its input with the previous token's (`shift`), whose input is kept per slot
    (`before`), and both sublayers may have a gate on their results (`gate_b`: its biases; the logits come with the projections)."""
    mixer: object
    norm1: torch.Tensor
    norm1b: torch.Tensor | None = None
    mlp: object = None
    norm2: torch.Tensor | None = None
    norm2b: torch.Tensor | None = None
    reinject: bool = False         # the embedding output is added to the residual stream before this layer
    shift: torch.Tensor | None = None
    before: torch.Tensor | None = None
    gate_b: tuple = (None, None)

    def again(self, reinject: bool = False) -> "MixerLayer":
        """A further run of the layer: the same weights, a state or cache of its own."""
        return replace(self, mixer=self.mixer.again(), reinject=reinject, before=None if self.before is None else torch.zeros_like(self.before))


@dataclass
class PostSum:
    """Layers are normed behind their sums, x <- norm(alpha x + y), and read x itself; a sinusoid of the position is added to the
    embedding. `freq`: its angular frequencies (float64)."""
    alpha: float
    freq: torch.Tensor


def sinusoid_frequencies(width: int, base: float = 10000.0) -> torch.Tensor:
    """Column 2i of a row is the sine, column 2i + 1 the cosine of position x frequency i."""
    return torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * torch.arange((width + 1) // 2, dtype=torch.float64) / width)


@dataclass
class MixerModel:
    """What `runtime.mixer_runtime.MixerRuntime` runs: an embedding, runs of layers, a final norm and an output matrix."""
    vocab: int
    width: int
    eps: float
    dtype: torch.dtype
    embed: torch.Tensor            # [vocab, width] bf16
    layers: list[MixerLayer]
    final_norm: torch.Tensor       # a factor on the logits is part of it
    head: FusedLinear
    plus_one: bool = True          # norm weights are stored around zero
    embed_scale: float = 1.0
    residual_scale: float = 1.0    # factor on every sublayer's output
    post: PostSum | None = None    # norms behind the sums instead of before the sublayers

    def windows(self) -> set[int]:
        return {L.mixer.window for L in self.layers if isinstance(L.mixer, LatentAttentionMixer)}


MIXERS = {"mlstm": MLSTMMixer, "gla": GLAMixer, "latent_attention": LatentAttentionMixer}
PAGED = {"latent_attention"}
