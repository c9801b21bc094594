"""Step function of mixer decoders: one call runs a mixed batch (portions of prompts of any size beside single decoded
tokens) from the states and pages that earlier calls left, and returns the logits that were asked for.

* Slots and pages come from `request_cache.RequestCache`; a request is admitted by its first entry and ends with `release`.
* Portions of up to `ROWS_MAX` tokens take the few-row kernels, longer ones the chunk / tensor-core kernels, in the same
  batch; the projections run over all rows together.
* A batch of single tokens is captured as a CUDA graph per batch size the second time it occurs; `decode_greedy` replays it
  with the tokens fed back on the device.

The single-request methods (`reset`, `prefill`, `decode_one`, `forward_logits`) are the token runtime that the generation
CLI and the servers expect of every model.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Sequence

import numpy as np
import torch

from ..models.mixer_layers import MixerModel, StepContext, Workspace
from ..ops import mixer_ops as mo
from .request_cache import RequestCache


@dataclass
class StepEntry:
    """A request's next tokens, and the places among them whose logits are wanted."""
    rid: object
    tokens: Sequence[int]
    want: Sequence[int] = field(default_factory=tuple)


def plan_portions(lengths: Sequence[int], starts: Sequence[int], slots: Sequence[int], windows: Sequence[int], rows_max: int = mo.ROWS_MAX,
                  chunk: int = mo.CHUNK, tile: int = 128) -> dict:
    """Index arrays (numpy int32) of a batch: per row its position, slot, (for a portion's last row) the slot again and how many
    tokens of its portion come after it, and the work lists of short and long portions. Pure host logic."""
    T = int(sum(lengths))
    pos, slot, last, behind = np.empty(T, np.int32), np.empty(T, np.int32), np.full(T, -1, np.int32), np.empty(T, np.int32)
    short, rows, long, chunks, chunk0, tiles, tile0 = [], [], [], [], [], [], []
    gather = {w: [] for w in windows}
    total = {w: 0 for w in windows}
    longest = {w: 0 for w in windows}
    r0 = 0
    for n, p0, s in zip(lengths, starts, slots):
        pos[r0:r0 + n] = np.arange(p0, p0 + n)
        slot[r0:r0 + n] = s
        last[r0 + n - 1] = s
        behind[r0:r0 + n] = np.arange(n - 1, -1, -1)
        seq = (r0, n, s, p0)
        if n <= rows_max:
            short.append(seq)
            rows.extend(range(r0, r0 + n))
        else:
            i = len(long)
            long.append(seq)
            chunk0.append(len(chunks))
            tile0.append(len(tiles))
            chunks += [(r0 + a, min(chunk, n - a), i, a // chunk) for a in range(0, n, chunk)]
            tiles += [(r0 + a, min(tile, n - a), i, 0) for a in range(0, n, tile)]
            for w in gather:
                first = max(0, p0 - w + 1) if w > 0 else 0
                gather[w].append((total[w], first))
                total[w] += p0 + n - first
                longest[w] = max(longest[w], p0 + n - first)
        r0 += n
    return {"T": T, "pos": pos, "slot": slot, "last": last, "behind": behind, "short": short, "rows": rows, "long": long, "chunks": chunks, "chunk0": chunk0,
            "tiles": tiles, "tile0": tile0, "gather": gather, "total": total, "longest": longest}


class _DecodeBatch:
    """Static inputs of the single-token step for one batch size, and its graph."""

    def __init__(self, n: int, device, vocab: int, hist: int):
        i32 = dict(dtype=torch.int32, device=device)
        self.n = n
        self.packed = torch.zeros(n * 8, **i32)              # seqs (4 n) | tokens | pos | slot | last: one copy per step
        self.seqs = self.packed[:4 * n].view(n, 4)
        self.tokens, self.pos, self.slot, self.last = (self.packed[(4 + k) * n:(5 + k) * n] for k in range(4))
        self.rows, self.behind = torch.arange(n, **i32), torch.zeros(n, **i32)
        self.hist = torch.zeros(n, hist, **i32)
        self.step = torch.zeros(1, **i32)
        self.cand_val, self.cand_idx = torch.zeros(n, 64, device=device), torch.zeros(n, 64, **i32)
        self.best_val, self.best = torch.zeros(n, device=device), torch.zeros(n, **i32)
        self.logits = None
        self.warm = False
        self.nodes = self.feed_nodes = 0
        self.graph = None          # forward + logits
        self.feed_warm = False
        self.feed_graph = None     # forward + logits + greedy pick + feedback


class MixerRuntime:
    HIST = 64

    def __init__(self, model: MixerModel, *, max_requests: int, pages: int, device: str = "cuda", use_graphs: bool = True):
        self.model, self.device, self.use_graphs = model, torch.device(device), use_graphs
        self.cache = RequestCache(max_requests, pages, mo.PAGE, device)
        self.ws, self.dec_ws = Workspace(device), Workspace(device)
        self.status = torch.zeros(1, dtype=torch.int32, device=device)
        self.max_requests, self.max_tokens = max_requests, pages * mo.PAGE
        self._windows = sorted(model.windows())
        self._dec: dict[int, _DecodeBatch] = {}
        self._pinned = torch.zeros(8 * max_requests, dtype=torch.int32).pin_memory()
        self._copied = torch.cuda.Event()
        self.launches = 0                          # kernels launched so far, graph nodes counted per replay
        self.launch_layers: list | None = None     # set to a list to collect the residual stream after every layer

    @property
    def vocab(self) -> int:
        return self.model.vocab

    # -- requests --------------------------------------------------------------------------
    def release(self, rid) -> None:
        self.cache.release(rid)

    def state_bytes(self) -> int:
        return sum(L.mixer.state_bytes() for L in self.model.layers if hasattr(L.mixer, "state_bytes"))

    def cache_bytes(self) -> int:
        return sum(L.mixer.cache_bytes() for L in self.model.layers if hasattr(L.mixer, "cache_bytes"))

    def check_status(self) -> None:
        """Raise when a bounded device wait of an earlier step ran out."""
        v = int(self.status.item())
        if v:
            self.status.zero_()
            raise RuntimeError(f"a kernel of the step gave up waiting (code {v})")

    # -- the step --------------------------------------------------------------------------
    @torch.no_grad()
    def step(self, entries: Sequence[StepEntry]) -> torch.Tensor:
        """Run the tokens of all entries as one batch; fp32 logits of the wanted places, in the order of the entries and of
        their `want`: [wanted, vocab] (valid until the next call)."""
        if not entries:
            return torch.empty(0, self.vocab, device=self.device)
        if len({e.rid for e in entries}) != len(entries):
            raise ValueError("a request occurs twice in one step")
        for e in entries:
            if not len(e.tokens):
                raise ValueError("an entry without tokens")
            if any(not 0 <= t < self.vocab for t in e.tokens):
                raise ValueError("token id outside the vocabulary")
            if any(not 0 <= w < len(e.tokens) for w in e.want):
                raise ValueError("a wanted place outside the entry's tokens")
        length = {e.rid: self.cache.length.get(e.rid, 0) for e in entries}
        self.cache.reserve({e.rid: length[e.rid] + len(e.tokens) for e in entries})
        self.cache.sync()
        if all(len(e.tokens) == 1 for e in entries) and len(entries) <= mo.ROWS_MAX:
            logits = self._decode(entries)
        else:
            n0 = mo.launches
            logits = self._mixed(entries)
            self.launches += mo.launches - n0
        for e in entries:
            self.cache.advance(e.rid, len(e.tokens))
        return logits

    def _forward(self, ctx: StepContext, want: torch.Tensor | None, n_want: int) -> torch.Tensor | None:
        """The model over one batch; logits of the rows in `want` (None: of every row)."""
        m, ws, T = self.model, ctx.ws, ctx.T
        if m.post is not None:
            return self._forward_post(ctx, want, n_want)
        hk = m.head.K                                                   # padded width of every sublayer's input
        x = ws.rows("x", T, m.width, torch.float32)
        h = ws.rows("h", T, hk, m.dtype)
        kw = dict(eps=m.eps, plus_one=m.plus_one)
        emb = dict(tokens=ctx.tokens, embed=m.embed, embed_scale=m.embed_scale)
        first = m.layers[0].norm1 if m.layers else None
        mo.sandwich_norm(x, w_pre=first, out=h, **emb, **kw)
        y: dict = {}                                                    # sublayer output that is still to be added to x
        kw["y_scale"] = m.residual_scale
        for i, L in enumerate(m.layers):
            if i:
                if self.launch_layers is not None:
                    mo.sandwich_norm(x, **y, **kw)
                    self.launch_layers.append(x.clone())
                    y = {}
                mo.sandwich_norm(x, w_pre=L.norm1, out=h, **y, **(dict(embed_add=True, **emb) if L.reinject else {}), **kw)
            y = dict(y=L.mixer.forward(ctx, h), w_post=L.norm1b)
            if L.mlp is not None:
                mo.sandwich_norm(x, w_pre=L.norm2, out=h, **y, **kw)
                y = dict(w_post=L.norm2b, **L.mlp.forward(ctx, h))
        if self.launch_layers is not None and y:
            mo.sandwich_norm(x, **y, **kw)
            self.launch_layers.append(x.clone())
            y = {}
        n = T if want is None else n_want
        if n == 0:
            return None
        hf = ws.rows("h_final", n, hk, m.dtype)
        mo.sandwich_norm(x, rows=want, count=n, w_pre=m.final_norm, out=hf, **y, **kw)
        return m.head(ctx, hf, "logits", torch.float32)

    def _forward_post(self, ctx: StepContext, want: torch.Tensor | None, n_want: int) -> torch.Tensor | None:
        """The same for a model whose norms follow the sums. The residual stream alternates between two buffers, since a step looks at
        the row before its own."""
        m, ws, T = self.model, ctx.ws, ctx.T
        hk, n = m.head.K, T if want is None else n_want
        old, new = ws.rows("x", T, m.width, torch.float32), ws.rows("x_other", T, m.width, torch.float32)
        h, hs, hf = ws.rows("h", T, hk, m.dtype), ws.rows("h_shift", T, hk, m.dtype), ws.rows("h_final", max(n, 1), hk, m.dtype)
        batch = dict(pos=ctx.pos.data_ptr(), slot=ctx.slot.data_ptr(), behind=ctx.behind.data_ptr(), M=T, width=m.width, ldo=hk,
                     out_f32=int(m.dtype == torch.float32), alpha=m.post.alpha, eps=m.eps)

        def entering(i: int) -> dict:                                   # what layer i reads
            L = m.layers[i]
            if L.shift is None:
                return dict(out=h)
            return dict(out=h, out_shift=hs, shift=L.shift, before=L.before)

        def step(**kw) -> None:
            nonlocal old, new
            y, gate = kw.get("y"), kw.get("gate")
            for name, key in (("y", "ldy"), ("y2", "ldy2"), ("gate", "ldg")):
                if kw.get(name) is not None:
                    kw[key] = kw[name].stride(0)
            if y is not None:
                kw.update(x=old, y_top=kw["y_rows"].shape[1] if "y_rows" in kw else 0)
            if gate is None:
                kw.pop("gate_b", None)
            mo.post_norm(mo.PostNorm(**{**batch, **{k: v.data_ptr() if isinstance(v, torch.Tensor) else v for k, v in kw.items()}}))
            old, new = new, old

        step(x_out=new, tokens=ctx.tokens, embed=m.embed, vocab=m.embed.shape[0], freq=m.post.freq, **entering(0))
        finished = False
        for i, L in enumerate(m.layers):
            last = i + 1 == len(m.layers)
            after = {} if last else entering(i + 1)
            y = dict(y=L.mixer.forward(ctx, h if L.shift is None else hs, h), w=L.norm1, gate_b=L.gate_b[0], save=L.before)
            if L.gate_b[0] is not None:
                y["gate"] = ws.rows("proj", T, L.mixer.proj.N, torch.float32)[:, L.mixer.proj.at["gate"]:]
            if L.mlp is None:
                step(x_out=new, **y, **after)
            else:
                step(x_out=new, out=h, **y)
                y = dict(w=L.norm2, gate_b=L.gate_b[1], **L.mlp.forward(ctx, h))
                if last and self.launch_layers is None:
                    finished = True
                    if n:
                        step(**y, rows=want, M=n, w_out=m.final_norm, out=hf)
                else:
                    step(x_out=new, **y, **after)
            if self.launch_layers is not None:
                self.launch_layers.append(old.clone())
        if n == 0:
            return None
        if not finished:
            mo.sandwich_norm(old, rows=want, count=n, w_pre=m.final_norm, out=hf, eps=m.eps, plus_one=False)
        return m.head(ctx, hf, "logits", torch.float32)

    def _mixed(self, entries: Sequence[StepEntry]) -> torch.Tensor:
        lens = [len(e.tokens) for e in entries]
        p = plan_portions(lens, [self.cache.length[e.rid] for e in entries], [self.cache.slot(e.rid) for e in entries], self._windows)
        want, r0 = [], 0
        for e in entries:
            want += [r0 + w for w in e.want]
            r0 += len(e.tokens)
        T = p["T"]
        parts: dict[str, tuple[int, int]] = {}
        arrays, off = [], 0

        def put(name, a):
            nonlocal off
            a = np.asarray(a, np.int32).reshape(-1)
            pad = -len(a) % 4                                           # every list starts on 16 bytes
            arrays.append(np.pad(a, (0, pad)))
            parts[name] = (off, len(a))
            off += len(a) + pad

        put("tokens", np.concatenate([np.asarray(e.tokens, np.int32) for e in entries]))
        for n in ("pos", "slot", "last", "behind", "short", "rows", "long", "chunks", "chunk0", "tiles", "tile0"):
            put(n, p[n])
        put("all", np.arange(T))
        put("want", want)
        for w in self._windows:
            put(f"gather{w}", p["gather"][w])
        dev = torch.from_numpy(np.concatenate(arrays)).to(self.device)
        at = lambda n: dev[parts[n][0]:parts[n][0] + parts[n][1]]
        ctx = StepContext(T, at("tokens"), at("pos"), at("slot"), at("last"), at("behind"), self.cache.device_table, self.ws, self.status,
                          short=at("short"), n_short=len(p["short"]), rows=at("rows"), n_rows=len(p["rows"]), all_rows=at("all"),
                          long=at("long"), n_long=len(p["long"]), chunks=at("chunks"), chunk0=at("chunk0"), n_chunks=len(p["chunks"]),
                          tiles=at("tiles"), n_tiles=len(p["tiles"]), tile0=at("tile0"),
                          gather={w: (at(f"gather{w}"), p["total"][w], p["longest"][w]) for w in self._windows})
        self.ws.trim()
        logits = self._forward(ctx, at("want"), len(want))
        if logits is None:
            return torch.empty(0, self.vocab, device=self.device)
        return logits[:, :self.vocab]

    # -- single-token batches --------------------------------------------------------------
    def _batch(self, n: int) -> _DecodeBatch:
        if n not in self._dec:
            self._dec[n] = _DecodeBatch(n, self.device, self.vocab, self.HIST)
        return self._dec[n]

    def _load_batch(self, b: _DecodeBatch, rids: Sequence, tokens: Sequence[int]) -> None:
        n = b.n
        self._copied.synchronize()                                      # the last copy out of the pinned buffer is done
        a = self._pinned.numpy()
        for i, (r, t) in enumerate(zip(rids, tokens)):
            s, q = self.cache.slot(r), self.cache.length[r]
            a[4 * i:4 * i + 4] = (i, 1, s, q)
            a[4 * n + i], a[5 * n + i], a[6 * n + i], a[7 * n + i] = t, q, s, s
        b.packed.copy_(self._pinned[:8 * n], non_blocking=True)
        self._copied.record()

    def _decode_forward(self, b: _DecodeBatch) -> torch.Tensor:
        ctx = StepContext(b.n, b.tokens, b.pos, b.slot, b.last, b.behind, self.cache.device_table, self.dec_ws, self.status, short=b.seqs, n_short=b.n,
                          rows=b.rows, n_rows=b.n, all_rows=b.rows)
        return self._forward(ctx, None, b.n)

    def _decode(self, entries: Sequence[StepEntry]) -> torch.Tensor:
        b, n0 = self._batch(len(entries)), mo.launches
        self._load_batch(b, [e.rid for e in entries], [int(e.tokens[0]) for e in entries])
        if not b.warm or not self.use_graphs or self.launch_layers is not None:
            b.logits, b.warm = self._decode_forward(b), True            # sizes every buffer of this batch size
            self.launches += mo.launches - n0
        else:
            if b.graph is None:
                torch.cuda.synchronize()
                b.graph = torch.cuda.CUDAGraph()
                with torch.cuda.graph(b.graph):
                    b.logits = self._decode_forward(b)
                b.nodes = mo.launches - n0
            b.graph.replay()
            self.launches += b.nodes
        want = [i for i, e in enumerate(entries) for _ in e.want]
        z = b.logits[:, :self.vocab]
        return z if want == list(range(b.n)) else z[want]

    def _feed_step(self, b: _DecodeBatch) -> None:
        b.logits = self._decode_forward(b)
        mo.argmax(b.logits, self.vocab, b.cand_val, b.cand_idx, b.best_val, b.best)
        mo.feed_tokens(b.best, b.tokens, b.pos, b.seqs, b.hist, b.step)

    @torch.no_grad()
    def decode_greedy(self, rids: Sequence, tokens: Sequence[int], steps: int) -> list[list[int]]:
        """`steps` greedy tokens of every request after its given next token, fed back on the device: [request][step]. Room for
        all of them is taken first."""
        if not 1 <= len(rids) <= mo.ROWS_MAX or not 1 <= steps <= self.HIST:
            raise ValueError("decode_greedy takes 1..8 requests and 1..64 steps")
        self.cache.reserve({r: self.cache.length.get(r, 0) + steps for r in rids})
        self.cache.sync()
        b = self._batch(len(rids))
        self._load_batch(b, rids, tokens)
        b.step.zero_()
        done, n0 = 0, mo.launches
        if not b.feed_warm or not self.use_graphs:
            self._feed_step(b)
            b.feed_warm, done = True, 1
            self.launches += mo.launches - n0
        if self.use_graphs and b.feed_graph is None and done < steps:
            torch.cuda.synchronize()
            n0 = mo.launches
            b.feed_graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(b.feed_graph):
                self._feed_step(b)
            b.feed_nodes = mo.launches - n0
        n0 = mo.launches
        for _ in range(done, steps):
            b.feed_graph.replay() if self.use_graphs else self._feed_step(b)
        self.launches += (steps - done) * b.feed_nodes if self.use_graphs else mo.launches - n0
        out = b.hist[:, :steps].tolist()
        for r in rids:
            self.cache.advance(r, steps)
        return out

    # -- token runtime of one request ---------------------------------------------------------
    _SINGLE = "single-request"

    def reset(self) -> None:
        if self._SINGLE in self.cache:
            self.cache.release(self._SINGLE)

    def forward_logits(self, tokens: Sequence[int]) -> torch.Tensor:
        """Feed tokens of the single request; logits of the last one [vocab]."""
        return self.step([StepEntry(self._SINGLE, list(tokens), (len(tokens) - 1,))])[0]

    def prefill(self, tokens: Sequence[int], portion: int = 2048) -> int:
        """The prompt in portions; the first greedy token."""
        z = None
        for a in range(0, len(tokens), portion):
            z = self.forward_logits(tokens[a:a + portion])
        return int(torch.argmax(z))

    def decode_one(self, token: int) -> int:
        return self.decode_greedy([self._SINGLE], [int(token)], 1)[0][0]
