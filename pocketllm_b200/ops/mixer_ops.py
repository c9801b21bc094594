"""Bindings of the mixer-decoder kernels: sandwich norms on an fp32 residual stream, fp32 and few-row bf16 linears, recurrent
outer-product states (gated linear attention, mLSTM), latent attention over a paged cache.

Every function launches on the current stream and writes into buffers its caller owns (so that a step can be captured in
a CUDA graph); a non-zero status raises.
"""
from __future__ import annotations

import ctypes
from ctypes import POINTER, Structure, byref, c_float, c_int, c_size_t, c_void_p

import torch

from . import EPI_BF16, EPI_F32, EPI_SWIGLU, _check
from . import lib as _lib

KIND_GLA, KIND_MLSTM = 0, 1
PAGE = 64           # tokens per cache page
CHUNK = 64          # tokens per chunk of the recurrent prefill form
ROWS_MAX = 8        # widest portion (and batch) of the few-row kernels


class StateMixer(Structure):
    """`PkStateMixer`: columns of the fused projection, constants, state and raw outputs of one recurrent layer."""
    _fields_ = [(n, c_void_p) for n in ("proj", "bi", "bf", "a2", "a2b", "S", "N", "Ms", "o", "nq", "m")] + \
               [(n, c_int) for n in ("kind", "ld", "oq", "ok", "ov", "og", "oi", "of", "oa", "H", "D", "V", "rank")] + \
               [(n, c_float) for n in ("qscale", "cap", "inv_tau")]


_sms: dict[int, int] = {}


def sm_count() -> int:
    d = torch.cuda.current_device()
    if d not in _sms:
        _sms[d] = torch.cuda.get_device_properties(d).multi_processor_count
    return _sms[d]


# argument kinds of the launchers, the stream excepted: p pointer, i int, f float
_SIGNATURES = {
    "pk_linear_f32": "pipiiiipi", "pk_linear_rows": "pipiiiipii", "pk_gemm_bf16": "pipiiiippippi",
    "pk_sandwich_norm": "pppipippiipifpii", "pk_feed_tokens": "pipppp" "ip", "pk_argmax": "piiiiipppp",
    "pk_state_rows": "ppi", "pk_state_chunks": "ppippip", "pk_state_out": "ppifpipii",
    "pk_latent_prep": "piiiiiiiipfpfpppp" "iiippi", "pk_latent_gather": "ppiippiip", "pk_latent_absorb": "piiiiiipipipi",
    "pk_latent_rows": "ppippppiiiiiifipp", "pk_latent_out": "ppiiiippipipi", "pk_latent_prefill": "pipipippiiiiifppip",
}
_bound: dict[tuple[int, str], object] = {}
_KERNELS = {"pk_state_chunks": 5, "pk_latent_out": 2, "pk_argmax": 2, "pk_feed_tokens": 2}     # launches per call, where not 1
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


def sandwich_norm(x: torch.Tensor, *, eps: float, out: torch.Tensor | None = None, w_pre: torch.Tensor | None = None,
                  tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None, y: torch.Tensor | None = None,
                  w_post: torch.Tensor | None = None, rows: torch.Tensor | None = None, count: int | None = None, plus_one: bool = True) -> None:
    """One step of the residual stream x [rows, width] fp32 (see sandwich_norm.cu). `rows`/`count`: norm only these rows."""
    M = (x.shape[0] if rows is None else rows.shape[0]) if count is None else count
    _call("pk_sandwich_norm", x, tokens, embed, 0 if embed is None else embed.shape[0], y, 0 if y is None else y.stride(0), w_post, rows, M,
          x.shape[1], w_pre, int(plus_one), eps, out, 0 if out is None else out.stride(0), int(out is not None and out.dtype == torch.float32))


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
    _call("pk_state_chunks", byref(d), seqs, nseq, chunks, chunk0, nchunks, ws)


def state_out(d: StateMixer, norm_w: torch.Tensor, per_head: bool, eps: float, last_slot: torch.Tensor, rows: int, out: torch.Tensor) -> None:
    """Head norm + output gate of `rows` rows; norm_w [H * V], or [V] when `per_head`."""
    _call("pk_state_out", byref(d), norm_w, int(per_head), eps, last_slot, rows, out, out.stride(0), int(out.dtype == torch.float32))


def latent_prep(proj: torch.Tensor, oq: int, oc: int, H: int, D: int, R: int, K: int, c_norm: torch.Tensor, eps: float, freq: torch.Tensor,
                mag: float, pos: torch.Tensor, slot: torch.Tensor, cache: torch.Tensor, table: torch.Tensor, qx: torch.Tensor | None,
                qf: torch.Tensor | None, qf_ld: int) -> None:
    _call("pk_latent_prep", proj, proj.stride(0), oq, oc, proj.shape[0], H, D, R, K, c_norm, eps, freq, mag, pos, slot, cache, table,
          table.stride(0), cache.shape[-1], int(cache.dtype == torch.float32), qx, qf, qf_ld)


def latent_gather(cache: torch.Tensor, table: torch.Tensor, seqs: torch.Tensor, gather: torch.Tensor, nseq: int, max_rows: int, out: torch.Tensor) -> None:
    _call("pk_latent_gather", cache, table, table.stride(0), cache.shape[-1], seqs, gather, nseq, max_rows, out)


def latent_absorb(proj: torch.Tensor, oq: int, H: int, D: int, R: int, K: int, uk: torch.Tensor, rows: torch.Tensor, nrows: int, qx: torch.Tensor,
                  row: int) -> None:
    _call("pk_latent_absorb", proj, proj.stride(0), oq, H, D, R, K, uk, int(uk.dtype == torch.float32), rows, nrows, qx, row)


def latent_rows(qx: torch.Tensor, rows: torch.Tensor, nrows: int, pos: torch.Tensor, slot: torch.Tensor, cache: torch.Tensor, table: torch.Tensor,
                H: int, K: int, window: int, scale: float, nsplit: int, part_o: torch.Tensor, part_ml: torch.Tensor) -> None:
    _call("pk_latent_rows", qx, rows, nrows, pos, slot, cache, table, table.stride(0), cache.shape[-1], int(cache.dtype == torch.float32), H, K,
          window, scale, nsplit, part_o, part_ml)


def latent_out(part_o: torch.Tensor, part_ml: torch.Tensor, nsplit: int, H: int, K: int, V: int, sink: torch.Tensor | None, rows: torch.Tensor,
               nrows: int, uv: torch.Tensor, out: torch.Tensor) -> None:
    _call("pk_latent_out", part_o, part_ml, nsplit, H, K, V, sink, rows, nrows, uv, int(uv.dtype == torch.float32), out, out.stride(0))


def latent_prefill(q: torch.Tensor, nrows: int, kv: torch.Tensor, kv_rows: int, tiles: torch.Tensor, ntiles: int, seqs: torch.Tensor,
                   gather: torch.Tensor, H: int, qk_panels: int, v_panels: int, V: int, window: int, scale: float, sink: torch.Tensor | None,
                   out: torch.Tensor, status: torch.Tensor) -> None:
    _call("pk_latent_prefill", q, nrows, kv, kv_rows, tiles, ntiles, seqs, gather, H, qk_panels, v_panels, V, window, scale, sink, out,
          out.stride(0), status)
