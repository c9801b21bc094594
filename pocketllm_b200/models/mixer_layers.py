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
        self.norm = _f32(w["norm"], device) if "norm" in w else None
        self.S = torch.zeros(slots, heads, dim, vdim, device=device)
        self.N = self.Ms = None
        a = self.proj.at
        self.keep: list[torch.Tensor] = []
        self.desc = dict(kind=kind, H=heads, D=dim, V=vdim, oq=a["q"], ok=a["k"], ov=a["v"], og=a["g"], qscale=dim ** -0.5, S=self.S.data_ptr())

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

    def again(self):
        o = copy.copy(self)
        o.cache = torch.zeros_like(self.cache)
        return o

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


class GroupedAttentionMixer:
    """Grouped-query attention over pages of [keys | values]: causal, in a window or in chunks (`mask`), rotary positions on a
    leading part of every query and key. With `diff` in its configuration a head has two softmax maps over the same values;
    its output is a1 - lambda a2, normed without a weight and scaled by 1 - diff. Long portions in bf16 run the tensor-core
    kernel on the pages, everything else the row kernel."""

    def __init__(self, w: dict, m: dict, eps: float, dtype, device, pages: int, context: int, mask: str = "window"):
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        diff = m.get("diff")
        maps = 1 if diff is None else 2
        if V > 512:
            raise ValueError("attention takes value dims up to 512")
        for n, r in (("q", H * maps * D), ("k", G * maps * D), ("v", G * V)):
            if w[n].shape[0] != r:
                raise ValueError(f"{n}: {w[n].shape[0]} rows, expected {r}")
        self.H, self.G, self.D, self.V, self.maps, self.dtype = H, G, D, V, maps, dtype
        self.proj = FusedLinear([("q", w["q"]), ("k", w["k"]), ("v", w["v"])], dtype, device)
        self.out = FusedLinear([("o", w["o"])], dtype, device)
        size = int((m.get("mask") or {}).get("size") or 0)
        self.span = min(size, context) if size else context         # most positions a query sees
        self.nsplit = max(1, min(64, (self.span + 31) // 32))
        dp, vp = pad_to(D, 8), pad_to(V, 8)
        self.row = G * (maps * dp + vp)
        self.q_ld = pad_to(D, 64)
        self.tensor_core = dtype == torch.bfloat16 and float(m["scale"]) > 0
        self.cache = torch.zeros(pages, mo.PAGE, self.row, dtype=dtype, device=device)
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        self.freq = rotary_frequencies(rot["dims"], rot["base"])[0].to(device)
        a = self.proj.at
        self.desc = dict(freq=self.freq.data_ptr() if rot["dims"] else None, oq=a["q"], ok=a["k"], ov=a["v"], H=H, G=G, maps=maps, D=D, V=V, R=rot["dims"],
                         dp=dp, vp=vp, row=self.row, f32=int(dtype == torch.float32), window=size if mask == "window" else 0,
                         chunk=size if mask == "chunk" else 0, q_ld=self.q_ld, scale=float(m["scale"]), eps=eps, post=1.0)
        if maps == 2:
            l = {n: w[n].double() for n in ("lq1", "lk1", "lq2", "lk2")}
            lam = float(torch.exp((l["lq1"] * l["lk1"]).sum()) - torch.exp((l["lq2"] * l["lk2"]).sum())) + float(diff)
            self.desc.update(lambda_=lam, head_norm=1, post=1.0 - float(diff))

    def again(self):
        o = copy.copy(self)
        o.cache = torch.zeros_like(self.cache)
        return o

    def cache_bytes(self) -> int:
        return self.cache.numel() * self.cache.element_size()

    def describe(self, ctx: StepContext, p: torch.Tensor, out: torch.Tensor) -> mo.PagedAttention:
        return mo.PagedAttention(proj=p.data_ptr(), ld=p.stride(0), pos=ctx.pos.data_ptr(), slot=ctx.slot.data_ptr(), cache=self.cache.data_ptr(),
                                 table=ctx.table.data_ptr(), table_ld=ctx.table.stride(0), out=out.data_ptr(), ldo=out.stride(0),
                                 status=ctx.status.data_ptr(), nsplit=1, **self.desc)

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        T, ws, nq = ctx.T, ctx.ws, self.H * self.maps
        p = self.proj(ctx, h, "proj", torch.float32)
        mix = ws.rows("mix", T, self.out.K, self.dtype)
        d = self.describe(ctx, p, mix)
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

    def forward(self, ctx: StepContext, h: torch.Tensor) -> tuple[torch.Tensor, None]:
        mid = ctx.ws.rows("mid", ctx.T, self.ff, self.dtype)
        mo.linear(h, self.gate_up, mid, ctx.status, swiglu=True)
        return self.down(ctx, mid, "y", torch.float32), None


class RoutedExperts:
    """Routed experts W_down max(W_up x, 0)^2. Few rows (and fp32) stream the chosen experts' weights; many rows are grouped by
    expert and multiplied on the tensor cores, and the sum over a token's experts is left to the norm that follows: `forward`
    returns rows and, per token, which of them to add."""

    def __init__(self, router_w: torch.Tensor, up: list[torch.Tensor], down: list[torch.Tensor], router: mo.Router, dtype, device):
        E, (ff, K), W = router.experts, up[0].shape, down[0].shape[0]
        self.route, self.W, self.dtype = router, W, dtype
        self.router = FusedLinear([("router", router_w)], dtype, device)
        self.ff, kp = pad_to(ff, 128), pad_to(K, 64)
        self.up = torch.zeros(E, self.ff, kp, dtype=dtype, device=device)
        self.down = torch.zeros(E, pad_to(W, 128), self.ff, dtype=dtype, device=device)
        for e in range(E):
            self.up[e, :ff, :K] = up[e].to(device=device, dtype=dtype)
            self.down[e, :W, :ff] = down[e].to(device=device, dtype=dtype)

    def forward(self, ctx: StepContext, h: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor | None]:
        T, ws, r = ctx.T, ctx.ws, self.route
        R = T * r.top
        z = self.router(ctx, h, "router", torch.float32)
        ids = ws.flat("route_ids", R, torch.int32)
        hidden = ws.rows("mid", R, self.ff, self.dtype)
        if T <= mo.ROWS_MAX or self.dtype == torch.float32:
            mo.expert_up_rows(r, z, h, self.up, ids, hidden)
            y = ws.rows("y", T, self.down.shape[1], torch.float32)
            mo.expert_down_rows(r, ids, hidden, self.down, self.W, y)
            return y, None
        place = ws.rows("route_place", T, r.top, torch.int32)
        seg, scale = ws.flat("route_seg", r.experts + 1, torch.int32), ws.flat("route_scale", R, torch.float32)
        x = ws.rows("route_x", R, self.up.shape[2], self.dtype)
        mo.expert_group(r, z, h, ids, ws.flat("route_w", R, torch.float32), seg, place, scale, x)
        mo.grouped_linear(x, self.up, seg, hidden, ctx.status, relu2=True, row_scale=scale, scale_after=r.on_output)
        y = ws.rows("expert_y", R, self.down.shape[1], torch.float32)
        mo.grouped_linear(hidden, self.down, seg, y, ctx.status)
        return y, place


@dataclass
class MixerLayer:
    """A mixer and an optional feed-forward, normed before and optionally (`norm1b`, `norm2b`) after."""
    mixer: object
    norm1: torch.Tensor
    norm1b: torch.Tensor | None = None
    mlp: object = None
    norm2: torch.Tensor | None = None
    norm2b: torch.Tensor | None = None
    reinject: bool = False         # the embedding output is added to the residual stream before this layer

    def again(self, reinject: bool) -> "MixerLayer":
        """A further run of the layer: the same weights, a state or cache of its own."""
        return replace(self, mixer=self.mixer.again(), reinject=reinject)


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

    def windows(self) -> set[int]:
        return {L.mixer.window for L in self.layers if isinstance(L.mixer, LatentAttentionMixer)}


MIXERS = {"mlstm": MLSTMMixer, "gla": GLAMixer, "latent_attention": LatentAttentionMixer}
PAGED = {"latent_attention"}
