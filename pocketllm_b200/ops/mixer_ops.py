"""Bindings of the mixer-decoder kernels: norms on an fp32 residual stream, fp32 and few-row bf16 linears, recurrent
outer-product states (gated linear attention, mLSTM, retention, state space, HGRN2), selective scan, latent and grouped-query attention over a
paged cache, routed experts.

Every function launches on the current stream and writes into buffers its caller owns (so that a step can be captured in
a CUDA graph); a non-zero status raises.
"""
from __future__ import annotations

from ctypes import POINTER, Structure, byref, c_float, c_int, c_size_t, c_void_p
from dataclasses import dataclass

import torch

from . import EPI_BF16, EPI_F32, EPI_SWIGLU, _check
from . import lib as _lib

KIND_GLA, KIND_MLSTM, KIND_RETENTION, KIND_SSD, KIND_HGRN = 0, 1, 2, 3, 4
SCORES = {"sigmoid": 0, "softmax": 1}      # router scores
EPI_RELU2 = 5       # grouped GEMM: squared ReLU with a factor per row
PAGE = 64           # tokens per cache page
CHUNK = 64          # tokens per chunk of the recurrent prefill form
ROWS_MAX = 8        # widest portion (and batch) of the few-row kernels


class StateMixer(Structure):
    """`PkStateMixer`: columns of the fused projection, constants, state and raw outputs of one recurrent layer."""
    _fields_ = [(n, c_void_p) for n in ("proj", "bi", "bf", "a2", "a2b", "S", "N", "Ms", "o", "nq", "m", "freq", "pw", "cw", "cb", "dtb", "A", "skip",
                                        "Cs", "low")] + \
               [(n, c_int) for n in ("kind", "ld", "oq", "ok", "ov", "og", "oi", "of", "oa", "H", "D", "V", "rank", "rot", "groups", "taps", "odt")] + \
               [(n, c_float) for n in ("qscale", "cap", "inv_tau")]


class PagedAttention(Structure):
    """`PkPagedAttention`: one grouped-query attention layer over one batch."""
    _fields_ = [(n, c_void_p) for n in ("proj", "freq", "pos", "slot", "cache", "table", "qx", "qf", "part_o", "part_ml", "out", "status", "q_norm", "k_norm",
                                        "sink", "v_first")] + \
               [(n, c_int) for n in ("ld", "oq", "ok", "ov", "H", "G", "maps", "D", "V", "R", "dp", "vp", "row", "table_ld", "f32", "window", "chunk", "q_ld",
                                     "ldo", "nsplit", "head_norm", "neighbours", "v_mix", "gate", "width")] + \
               [(n, c_float) for n in ("scale", "lambda_", "post", "eps", "cap", "mix")]


class SelectiveScan(Structure):
    """`PkSelectiveScan`: one selective-scan layer over one batch."""
    _fields_ = [(n, c_void_p) for n in ("proj", "xc", "dbc", "dt", "w_dt", "dt_bias", "A", "skip", "cw", "cb", "S", "ring", "out", "pos", "slot")] + \
               [(n, c_int) for n in ("ld", "ox", "oz", "ldx", "ldb", "ldt", "ldw", "ldo", "oB", "oC", "inner", "N", "rank", "taps", "f32")]


class PostNorm(Structure):
    """`PkPostNorm`: one residual step with its norm behind the sum."""
    _fields_ = [(n, c_void_p) for n in ("x", "x_out", "tokens", "embed", "freq", "y", "y_rows", "y2", "gate", "gate_b", "w", "w_out", "pos", "slot", "behind", "save",
                                        "shift", "before", "rows", "out", "out_shift")] + \
               [(n, c_int) for n in ("vocab", "ldy", "y_top", "ldy2", "ldg", "M", "width", "ldo", "out_f32")] + [(n, c_float) for n in ("alpha", "eps")]


_sms: dict[int, int] = {}


def sm_count() -> int:
    d = torch.cuda.current_device()
    if d not in _sms:
        _sms[d] = torch.cuda.get_device_properties(d).multi_processor_count
    return _sms[d]


# argument kinds of the launchers, the stream excepted: p pointer, i int, f float
_SIGNATURES = {
    "pk_linear_f32": "pipiiiipi", "pk_linear_rows": "pipiiiipii", "pk_linear_rows2": "ppiipiiiipii", "pk_gemm_bf16": "pipiiiippippi",
    "pk_sandwich_norm": "pppifipipifpiippp" "iipifpii", "pk_feed_tokens": "pipppp" "ip", "pk_post_norm": "p", "pk_argmax": "piiiiipppp",
    "pk_state_rows": "ppi", "pk_state_chunks": "ppippip", "pk_state_out": "ppifpipii", "pk_ssd_out": "ppifpppipiii", "pk_ssd_tiles": "ppippipp", "pk_ssd_rows": "ppii",
    "pk_scan_conv": "pi", "pk_scan_split": "piiiip", "pk_scan_rows": "ppi", "pk_scan_tiles": "ppi",
    "pk_latent_prep": "piiiiiiiipfpfpppp" "iiippi" "ippi", "pk_latent_gather": "ppiippiip", "pk_latent_absorb": "piiiiiipipipii",
    "pk_latent_rows": "ppippppiiiiiifipp", "pk_latent_out": "ppiiiippipipipi", "pk_latent_prefill": "pipipippiiiiifppipip",
    "pk_paged_prep": "pi", "pk_paged_rows": "ppi", "pk_paged_merge": "ppi", "pk_paged_prefill": "piipip",
    "pk_expert_up_rows": "piiiiifppipiipiipiiippii", "pk_expert_down_rows": "piipiipiiiipii", "pk_expert_group": "piiiiifppipipppppp" "iip",
    "pk_gemm_bf16_grouped_scaled": "pippiiiiipipipi",
}
_bound: dict[tuple[int, str], object] = {}
_KERNELS = {"pk_state_chunks": 5, "pk_ssd_tiles": 4, "pk_latent_out": 2, "pk_argmax": 2, "pk_feed_tokens": 2, "pk_expert_group": 3}     # launches per call, where not 1
launches = 0        # kernels launched (or captured) by this process through `_call`


def _call(name: str, *args) -> None:
    """Launch `name` on the current stream; tensors are passed as their address."""
    global launches
    k = _lib.kernels()
    f = _bound.get((id(k), name))
    if f is None:
        f = k[name]          # a function object of its own: other modules call the shared one without a prototype
        f.argtypes = [{"p": c_void_p, "i": c_int, "f": c_float}[c] for c in _SIGNATURES[name]] + [c_void_p]
        _bound[(id(k), name)] = f
    a = [x.data_ptr() if isinstance(x, torch.Tensor) else x for x in args]
    launches += _KERNELS.get(name, 1)
    st = f(*a, torch.cuda.current_stream().cuda_stream)
    if st != 0:
        _check(st, name)


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, status: torch.Tensor, *, swiglu: bool = False) -> torch.Tensor:
    """out[M, :] = x[M, K] w[N, K]^T. fp32 x: fp32 arithmetic. bf16 x: weight streaming up to eight rows, the tcgen05 GEMM
    beyond (K a multiple of 64); `out` bf16 or fp32. `swiglu`: w holds gate rows, then as many up rows."""
    M, K = x.shape
    N = w.shape[0]
    if x.dtype == torch.float32:
        _call("pk_linear_f32", x, x.stride(0), w, M, N, K, int(swiglu), out, out.stride(0))
        return out
    f32 = out.dtype == torch.float32
    if M <= ROWS_MAX:
        epi = 1 if swiglu else 2 if f32 else 0
        _call("pk_linear_rows", x, x.stride(0), w, M, N, K, epi, out, out.stride(0), sm_count())
    else:
        epi = EPI_SWIGLU if swiglu else EPI_F32 if f32 else EPI_BF16
        _call("pk_gemm_bf16", x, x.stride(0), w, M, N, K, epi, out, None, out.stride(0), status, None, sm_count())
    return out


def linear2(x: torch.Tensor, x2: torch.Tensor, split: int, w: torch.Tensor, out: torch.Tensor, status: torch.Tensor) -> torch.Tensor:
    """As `linear` (fp32 out), with `x2` as the input of the weight rows from `split` on; one launch up to eight rows of bf16."""
    M, K = x.shape
    if x.dtype == torch.float32 or M > ROWS_MAX:
        linear(x, w[:split], out[:, :split], status)
        linear(x2, w[split:], out[:, split:], status)
    else:
        _call("pk_linear_rows2", x, x2, split, x.stride(0), w, M, w.shape[0], K, 2, out, out.stride(0), sm_count())
    return out


def sandwich_norm(x: torch.Tensor, *, eps: float, out: torch.Tensor | None = None, w_pre: torch.Tensor | None = None,
                  tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None, embed_scale: float = 1.0, embed_add: bool = False,
                  y: torch.Tensor | None = None, y_rows: torch.Tensor | None = None, y_scale: float = 1.0, skip: torch.Tensor | None = None,
                  skip_w: torch.Tensor | None = None, w_post: torch.Tensor | None = None, rows: torch.Tensor | None = None, count: int | None = None,
                  plus_one: bool = True) -> None:
    """One step of the residual stream x [rows, width] fp32 (see sandwich_norm.cu). `rows`/`count`: norm only these rows; `y_rows`
    [rows, n]: a row's y is the sum of these n rows of `y` (negative: none); `skip_w` [rows] x the row of `skip` is part of y; y is
    multiplied by `y_scale`; `embed_add`: the scaled embedding row is added instead of starting x."""
    M = (x.shape[0] if rows is None else rows.shape[0]) if count is None else count
    _call("pk_sandwich_norm", x, tokens, embed, 0 if embed is None else embed.shape[0], embed_scale, int(embed_add), y, 0 if y is None else y.stride(0),
          y_rows, 0 if y_rows is None else y_rows.shape[1], y_scale, skip, 0 if skip is None else skip.stride(0),
          int(skip is not None and skip.dtype == torch.float32), skip_w, w_post, rows, M, x.shape[1], w_pre, int(plus_one), eps, out,
          0 if out is None else out.stride(0), int(out is not None and out.dtype == torch.float32))


def post_norm(d: PostNorm) -> None:
    """One step of a residual stream that is normed behind the sum (see post_norm.cu)."""
    _call("pk_post_norm", byref(d))


def feed_tokens(nxt: torch.Tensor, tokens: torch.Tensor, pos: torch.Tensor, seqs: torch.Tensor, hist: torch.Tensor, step: torch.Tensor) -> None:
    """Greedy feedback on the device: nxt [n] becomes the rows' input token, positions advance, hist[row, step] keeps it."""
    _call("pk_feed_tokens", nxt, nxt.shape[0], tokens, pos, seqs, hist, hist.stride(0), step)


def argmax(logits: torch.Tensor, n: int, cand_val: torch.Tensor, cand_idx: torch.Tensor, out_val: torch.Tensor, out_idx: torch.Tensor) -> None:
    """Greedy pick of every row of logits [M, ld] over its first n columns (lowest id on ties)."""
    M = logits.shape[0]
    nb = cand_val.shape[1]
    _call("pk_argmax", logits, logits.stride(0), M, n, 0, nb, cand_val, cand_idx, out_val, out_idx)


def state_rows(d: StateMixer, seqs: torch.Tensor, nseq: int) -> None:
    _call("pk_state_rows", byref(d), seqs, nseq)


def state_chunk_workspace(d: StateMixer, nchunks: int) -> int:
    fn = _lib.kernels().pk_state_chunk_workspace
    fn.restype = c_size_t
    fn.argtypes = [POINTER(StateMixer), c_int]
    return int(fn(byref(d), nchunks))


def state_chunks(d: StateMixer, seqs: torch.Tensor, nseq: int, chunks: torch.Tensor, chunk0: torch.Tensor, nchunks: int, ws: torch.Tensor) -> None:
    global launches
    _call("pk_state_chunks", byref(d), seqs, nseq, chunks, chunk0, nchunks, ws)
    launches -= int(d.kind in (KIND_RETENTION, KIND_HGRN))      # no gates


def state_out(d: StateMixer, norm_w: torch.Tensor | None, per_head: bool, eps: float, last_slot: torch.Tensor, rows: int, out: torch.Tensor) -> None:
    """Head norm + output gate of `rows` rows; norm_w [H * V], [V] when `per_head`, or None."""
    _call("pk_state_out", byref(d), norm_w, int(per_head), eps, last_slot, rows, out, out.stride(0), int(out.dtype == torch.float32))


def ssd_rows(d: StateMixer, seqs: torch.Tensor, nseq: int) -> None:
    """Recurrence of short portions of a state-space layer, its convolution included."""
    _call("pk_ssd_rows", byref(d), seqs, nseq, sm_count())


def ssd_tile_workspace(d: StateMixer, ntiles: int) -> int:
    """Workspace floats of `ssd_tiles`; 0: the shape does not fit it."""
    fn = _lib.kernels().pk_ssd_tile_workspace
    fn.restype, fn.argtypes = c_size_t, [POINTER(StateMixer), c_int]
    return int(fn(byref(d), ntiles))


def ssd_tiles(d: StateMixer, seqs: torch.Tensor, nseq: int, tiles: torch.Tensor, tile0: torch.Tensor, ntiles: int, ws: torch.Tensor,
              status: torch.Tensor) -> None:
    """Recurrence of long portions on the tensor cores, in tiles of 128 tokens."""
    _call("pk_ssd_tiles", byref(d), seqs, nseq, tiles, tile0, ntiles, ws, status)


def ssd_out(d: StateMixer, norm_w: torch.Tensor, parts: int, eps: float, slots: torch.Tensor, behind: torch.Tensor, pos: torch.Tensor, rows: int,
            out: torch.Tensor) -> None:
    """Gate and norm of a state-space layer, the ring of its convolution; `out` [rows, columns of this layer] (a view is fine)."""
    _call("pk_ssd_out", byref(d), norm_w, parts, eps, slots, behind, pos, rows, out, out.stride(0), out.shape[1], int(out.dtype == torch.float32))


def scan_conv(d: SelectiveScan, rows: int) -> None:
    """Convolution and SiLU of a selective-scan layer, all rows of a step."""
    _call("pk_scan_conv", byref(d), rows)


def scan_split(d: torch.Tensor, rank: int, out: torch.Tensor) -> None:
    """The first `rank` columns of d (fp32) as two bf16 terms side by side, out [rows, 2 x padded rank]."""
    _call("pk_scan_split", d, d.stride(0), rank, out.shape[1] // 2, out.shape[0], out)


def scan_rows(d: SelectiveScan, seqs: torch.Tensor, nseq: int) -> None:
    """Recurrence, gate and ring of short portions, W_dt included."""
    _call("pk_scan_rows", byref(d), seqs, nseq)


def scan_tiles(d: SelectiveScan, seqs: torch.Tensor, nseq: int) -> None:
    """Recurrence, gate and ring of long portions."""
    _call("pk_scan_tiles", byref(d), seqs, nseq)


def latent_prep(proj: torch.Tensor, oq: int, oc: int, H: int, D: int, R: int, K: int, c_norm: torch.Tensor, eps: float, freq: torch.Tensor,
                mag: float, pos: torch.Tensor, slot: torch.Tensor, cache: torch.Tensor, table: torch.Tensor, qx: torch.Tensor | None,
                qf: torch.Tensor | None, qf_ld: int, *, q_rank: int = 0, q_norm: torch.Tensor | None = None, ql: torch.Tensor | None = None) -> None:
    """`q_rank`: the columns at `oq` are the queries' latent, normed into `ql` [rows, padded rank]."""
    _call("pk_latent_prep", proj, proj.stride(0), oq, oc, proj.shape[0], H, D, R, K, c_norm, eps, freq, mag, pos, slot, cache, table,
          table.stride(0), cache.shape[-1], int(cache.dtype == torch.float32), qx, qf, qf_ld, q_rank, q_norm, ql, 0 if ql is None else ql.shape[1])


def latent_gather(cache: torch.Tensor, table: torch.Tensor, seqs: torch.Tensor, gather: torch.Tensor, nseq: int, max_rows: int, out: torch.Tensor) -> None:
    _call("pk_latent_gather", cache, table, table.stride(0), cache.shape[-1], seqs, gather, nseq, max_rows, out)


def latent_absorb(proj: torch.Tensor, oq: int, H: int, D: int, R: int, K: int, uk: torch.Tensor, rows: torch.Tensor, nrows: int, qx: torch.Tensor,
                  row: int, k_pad: int | None = None) -> None:
    """`R`: query columns between the heads' unrotated parts; columns K .. `k_pad` of qx are set to zero."""
    _call("pk_latent_absorb", proj, proj.stride(0), oq, H, D, R, K, uk, int(uk.dtype == torch.float32), rows, nrows, qx, row, k_pad or K)


def latent_rows(qx: torch.Tensor, rows: torch.Tensor, nrows: int, pos: torch.Tensor, slot: torch.Tensor, cache: torch.Tensor, table: torch.Tensor,
                H: int, K: int, window: int, scale: float, nsplit: int, part_o: torch.Tensor, part_ml: torch.Tensor) -> None:
    _call("pk_latent_rows", qx, rows, nrows, pos, slot, cache, table, table.stride(0), cache.shape[-1], int(cache.dtype == torch.float32), H, K,
          window, scale, nsplit, part_o, part_ml)


def latent_out(part_o: torch.Tensor, part_ml: torch.Tensor, nsplit: int, H: int, K: int, V: int, sink: torch.Tensor | None, rows: torch.Tensor,
               nrows: int, uv: torch.Tensor, out: torch.Tensor, gate: torch.Tensor | None = None) -> None:
    _call("pk_latent_out", part_o, part_ml, nsplit, H, K, V, sink, rows, nrows, uv, int(uv.dtype == torch.float32), out, out.stride(0), gate,
          0 if gate is None else gate.stride(0))


def latent_prefill(q: torch.Tensor, nrows: int, kv: torch.Tensor, kv_rows: int, tiles: torch.Tensor, ntiles: int, seqs: torch.Tensor,
                   gather: torch.Tensor, H: int, qk_panels: int, v_panels: int, V: int, window: int, scale: float, sink: torch.Tensor | None,
                   out: torch.Tensor, status: torch.Tensor, gate: torch.Tensor | None = None) -> None:
    _call("pk_latent_prefill", q, nrows, kv, kv_rows, tiles, ntiles, seqs, gather, H, qk_panels, v_panels, V, window, scale, sink, out,
          out.stride(0), gate, 0 if gate is None else gate.stride(0), status)


def paged_prep(a: PagedAttention, rows: int) -> None:
    """Rotation, cache append and queries of all rows of a step."""
    _call("pk_paged_prep", byref(a), rows)


def paged_rows(a: PagedAttention, rows: torch.Tensor, nrows: int) -> None:
    """Partial attention of the listed rows (splits into part_o / part_ml)."""
    _call("pk_paged_rows", byref(a), rows, nrows)


def paged_merge(a: PagedAttention, rows: torch.Tensor | None, nrows: int) -> None:
    """Splits (or finished fp32 outputs) of the listed rows -> head outputs."""
    _call("pk_paged_merge", byref(a), rows, nrows)


def paged_prefill_form(maps: int, D: int, V: int) -> int:
    """What the tensor-core kernel does with this shape: 1 finished outputs, 0 fp32 outputs for `paged_merge`, -1 nothing."""
    fn = _lib.kernels().pk_paged_prefill_form
    fn.restype, fn.argtypes = c_int, [c_int, c_int, c_int]
    return int(fn(maps, D, V))


def paged_prefill(a: PagedAttention, rows: int, pages: int, tiles: torch.Tensor, ntiles: int, seqs: torch.Tensor) -> None:
    _call("pk_paged_prefill", byref(a), rows, pages, tiles, ntiles, seqs)


@dataclass(frozen=True)
class Router:
    """How experts are chosen and weighted from router logits."""
    experts: int
    top: int
    score: str = "sigmoid"
    renorm: bool = False        # chosen weights divided by their sum
    scale: float = 1.0
    on_output: bool = False     # the weight multiplies an expert's output instead of its input
    identity: int = 0           # experts behind the others that return their input

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    def args(self, correction: torch.Tensor | None, skip_w: torch.Tensor | None, bias: torch.Tensor | None) -> tuple:
        return self.outputs, self.top, SCORES[self.score], int(self.renorm), self.scale, correction, bias, self.identity, skip_w


def expert_up_rows(r: Router, logits: torch.Tensor, x: torch.Tensor, w: torch.Tensor, ids: torch.Tensor, hidden: torch.Tensor, *, gated: bool = False,
                   correction: torch.Tensor | None = None, skip_w: torch.Tensor | None = None,
                   bias: torch.Tensor | None = None) -> None:
    """hidden [T * top, N] = squared ReLU of the chosen experts' up products, w [experts, N, K]; `gated`: silu(gate) * up, w [experts, N
    gate rows and N up rows, K]. ids [T * top] out; `correction` [outputs] counts for the choice, `bias` [outputs] is part of the
    logits; skip_w [T] out (identities)."""
    E, N, K = w.shape
    _call("pk_expert_up_rows", logits, logits.stride(0), *r.args(correction, skip_w, bias), int(r.on_output), int(gated), x, x.stride(0), x.shape[0], w,
          N // 2 if gated else N, K, int(w.dtype == torch.float32), ids, hidden, hidden.stride(0), sm_count())


def expert_down_rows(r: Router, ids: torch.Tensor, hidden: torch.Tensor, w: torch.Tensor, n: int, y: torch.Tensor) -> None:
    """y [T, n] fp32 = sum over a token's experts of w[expert, :n] . hidden; w [experts, rows, K]."""
    E, rows, K = w.shape
    _call("pk_expert_down_rows", ids, r.top, r.experts, hidden, hidden.stride(0), y.shape[0], w, n, rows, K, int(w.dtype == torch.float32), y, y.stride(0),
          sm_count())


def expert_group(r: Router, logits: torch.Tensor, x: torch.Tensor, ids: torch.Tensor, weights: torch.Tensor, seg: torch.Tensor, place: torch.Tensor,
                 row_scale: torch.Tensor, rows: torch.Tensor, *, correction: torch.Tensor | None = None, skip_w: torch.Tensor | None = None,
                   bias: torch.Tensor | None = None) -> None:
    """Routes of the tokens grouped by expert, token rows gathered in that order (rows [T * top, K])."""
    _call("pk_expert_group", logits, logits.stride(0), *r.args(correction, skip_w, bias), x.shape[0], ids, weights, seg, place, row_scale, x, x.stride(0),
          rows.shape[1], rows)


def grouped_linear(x: torch.Tensor, w: torch.Tensor, seg: torch.Tensor, out: torch.Tensor, status: torch.Tensor, *, relu2: bool = False,
                   swiglu: bool = False, row_scale: torch.Tensor | None = None, scale_after: bool = False) -> None:
    """out rows of group g = x rows . w[g]^T on the tensor cores (x, w bf16; w [groups, N, K], N a multiple of 128, K of 64); fp32 out,
    or bf16 squared ReLU, or SwiGLU (N / 2 gate rows, then N / 2 up rows) with a factor per row."""
    G, N, K = w.shape
    _call("pk_gemm_bf16_grouped_scaled", x, x.stride(0), w, seg, G, x.shape[0], N, K, EPI_RELU2 if relu2 else EPI_SWIGLU if swiglu else EPI_F32, out, out.stride(0), row_scale,
          int(scale_after), status, sm_count())
