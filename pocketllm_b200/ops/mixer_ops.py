"""Bindings of the mixer-decoder kernels: sandwich norms on an fp32 residual stream, fp32 and few-row bf16 linears, recurrent
outer-product states (gated linear attention, mLSTM), latent attention over a paged cache.

Every function launches on the current stream and writes into buffers its caller owns (so that a step can be captured in
a CUDA graph); a non-zero status raises.
"""
from __future__ import annotations

import ctypes
from ctypes import POINTER, Structure, byref, c_float, c_int, c_size_t, c_void_p

import torch

from . import EPI_BF16, EPI_F32, EPI_SWIGLU, _check, _ptr, _stream
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


def _k():
    return _lib.kernels()


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, status: torch.Tensor, *, swiglu: bool = False) -> torch.Tensor:
    """out[M, :] = x[M, K] w[N, K]^T. fp32 x: fp32 arithmetic. bf16 x: weight streaming up to eight rows, the tcgen05 GEMM
    beyond (K a multiple of 64); `out` bf16 or fp32. `swiglu`: w holds gate rows, then as many up rows."""
    M, K = x.shape
    N = w.shape[0]
    if x.dtype == torch.float32:
        _check(_k().pk_linear_f32(_ptr(x), c_int(x.stride(0)), _ptr(w), c_int(M), c_int(N), c_int(K), c_int(int(swiglu)), _ptr(out),
                                  c_int(out.stride(0)), _stream()), "pk_linear_f32")
        return out
    f32 = out.dtype == torch.float32
    if M <= ROWS_MAX:
        epi = 1 if swiglu else 2 if f32 else 0
        _check(_k().pk_linear_rows(_ptr(x), c_int(x.stride(0)), _ptr(w), c_int(M), c_int(N), c_int(K), c_int(epi), _ptr(out),
                                   c_int(out.stride(0)), c_int(sm_count()), _stream()), "pk_linear_rows")
    else:
        epi = EPI_SWIGLU if swiglu else EPI_F32 if f32 else EPI_BF16
        _check(_k().pk_gemm_bf16(_ptr(x), c_int(x.stride(0)), _ptr(w), c_int(M), c_int(N), c_int(K), c_int(epi), _ptr(out), c_void_p(0),
                                 c_int(out.stride(0)), _ptr(status), c_void_p(0), c_int(sm_count()), _stream()), "pk_gemm_bf16")
    return out


def sandwich_norm(x: torch.Tensor, *, eps: float, out: torch.Tensor | None = None, w_pre: torch.Tensor | None = None,
                  tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None, y: torch.Tensor | None = None,
                  w_post: torch.Tensor | None = None, rows: torch.Tensor | None = None, count: int | None = None, plus_one: bool = True) -> None:
    """One step of the residual stream x [rows, width] fp32 (see sandwich_norm.cu). `rows`/`count`: norm only these rows."""
    M = (x.shape[0] if rows is None else rows.shape[0]) if count is None else count
    _check(_k().pk_sandwich_norm(
        _ptr(x), _ptr(tokens), _ptr(embed), c_int(0 if embed is None else embed.shape[0]), _ptr(y), c_int(0 if y is None else y.stride(0)),
        _ptr(w_post), _ptr(rows), c_int(M), c_int(x.shape[1]), _ptr(w_pre), c_int(int(plus_one)), c_float(eps), _ptr(out),
        c_int(0 if out is None else out.stride(0)), c_int(int(out is not None and out.dtype == torch.float32)), _stream()), "pk_sandwich_norm")


def feed_tokens(nxt: torch.Tensor, tokens: torch.Tensor, pos: torch.Tensor, seqs: torch.Tensor, hist: torch.Tensor, step: torch.Tensor) -> None:
    """Greedy feedback on the device: nxt [n] becomes the rows' input token, positions advance, hist[row, step] keeps it."""
    _check(_k().pk_feed_tokens(_ptr(nxt), c_int(nxt.shape[0]), _ptr(tokens), _ptr(pos), _ptr(seqs), _ptr(hist), c_int(hist.stride(0)), _ptr(step),
                               _stream()), "pk_feed_tokens")


def argmax(logits: torch.Tensor, n: int, cand_val: torch.Tensor, cand_idx: torch.Tensor, out_val: torch.Tensor, out_idx: torch.Tensor) -> None:
    """Greedy pick of every row of logits [M, ld] over its first n columns (lowest id on ties)."""
    M = logits.shape[0]
    nb = cand_val.shape[1]
    _check(_k().pk_argmax(_ptr(logits), c_int(logits.stride(0)), c_int(M), c_int(n), c_int(0), c_int(nb), _ptr(cand_val), _ptr(cand_idx),
                          _ptr(out_val), _ptr(out_idx), _stream()), "pk_argmax")


def state_rows(d: StateMixer, seqs: torch.Tensor, nseq: int) -> None:
    _check(_k().pk_state_rows(byref(d), _ptr(seqs), c_int(nseq), _stream()), "pk_state_rows")


def state_chunk_workspace(d: StateMixer, nchunks: int) -> int:
    fn = _k().pk_state_chunk_workspace
    fn.restype = c_size_t
    fn.argtypes = [POINTER(StateMixer), c_int]
    return int(fn(byref(d), nchunks))


def state_chunks(d: StateMixer, seqs: torch.Tensor, nseq: int, chunks: torch.Tensor, chunk0: torch.Tensor, nchunks: int, ws: torch.Tensor) -> None:
    _check(_k().pk_state_chunks(byref(d), _ptr(seqs), c_int(nseq), _ptr(chunks), _ptr(chunk0), c_int(nchunks), _ptr(ws), _stream()), "pk_state_chunks")


def state_out(d: StateMixer, norm_w: torch.Tensor, per_head: bool, eps: float, last_slot: torch.Tensor, rows: int, out: torch.Tensor) -> None:
    """Head norm + output gate of `rows` rows; norm_w [H * V], or [V] when `per_head`."""
    _check(_k().pk_state_out(byref(d), _ptr(norm_w), c_int(int(per_head)), c_float(eps), _ptr(last_slot), c_int(rows), _ptr(out),
                             c_int(out.stride(0)), c_int(int(out.dtype == torch.float32)), _stream()), "pk_state_out")


def latent_prep(proj: torch.Tensor, oq: int, oc: int, H: int, D: int, R: int, K: int, c_norm: torch.Tensor, eps: float, freq: torch.Tensor,
                mag: float, pos: torch.Tensor, slot: torch.Tensor, cache: torch.Tensor, table: torch.Tensor, qx: torch.Tensor | None,
                qf: torch.Tensor | None, qf_ld: int) -> None:
    _check(_k().pk_latent_prep(
        _ptr(proj), c_int(proj.stride(0)), c_int(oq), c_int(oc), c_int(proj.shape[0]), c_int(H), c_int(D), c_int(R), c_int(K), _ptr(c_norm),
        c_float(eps), _ptr(freq), c_float(mag), _ptr(pos), _ptr(slot), _ptr(cache), _ptr(table), c_int(table.stride(0)), c_int(cache.shape[-1]),
        c_int(int(cache.dtype == torch.float32)), _ptr(qx), _ptr(qf), c_int(qf_ld), _stream()), "pk_latent_prep")


def latent_gather(cache: torch.Tensor, table: torch.Tensor, seqs: torch.Tensor, gather: torch.Tensor, nseq: int, max_rows: int, out: torch.Tensor) -> None:
    _check(_k().pk_latent_gather(_ptr(cache), _ptr(table), c_int(table.stride(0)), c_int(cache.shape[-1]), _ptr(seqs), _ptr(gather), c_int(nseq),
                                 c_int(max_rows), _ptr(out), _stream()), "pk_latent_gather")


def latent_absorb(proj: torch.Tensor, oq: int, H: int, D: int, R: int, K: int, uk: torch.Tensor, rows: torch.Tensor, nrows: int, qx: torch.Tensor,
                  row: int) -> None:
    _check(_k().pk_latent_absorb(_ptr(proj), c_int(proj.stride(0)), c_int(oq), c_int(H), c_int(D), c_int(R), c_int(K), _ptr(uk),
                                 c_int(int(uk.dtype == torch.float32)), _ptr(rows), c_int(nrows), _ptr(qx), c_int(row), _stream()), "pk_latent_absorb")


def latent_rows(qx: torch.Tensor, rows: torch.Tensor, nrows: int, pos: torch.Tensor, slot: torch.Tensor, cache: torch.Tensor, table: torch.Tensor,
                H: int, K: int, window: int, scale: float, nsplit: int, part_o: torch.Tensor, part_ml: torch.Tensor) -> None:
    _check(_k().pk_latent_rows(_ptr(qx), _ptr(rows), c_int(nrows), _ptr(pos), _ptr(slot), _ptr(cache), _ptr(table), c_int(table.stride(0)),
                               c_int(cache.shape[-1]), c_int(int(cache.dtype == torch.float32)), c_int(H), c_int(K), c_int(window), c_float(scale),
                               c_int(nsplit), _ptr(part_o), _ptr(part_ml), _stream()), "pk_latent_rows")


def latent_out(part_o: torch.Tensor, part_ml: torch.Tensor, nsplit: int, H: int, K: int, V: int, sink: torch.Tensor | None, rows: torch.Tensor,
               nrows: int, uv: torch.Tensor, out: torch.Tensor) -> None:
    _check(_k().pk_latent_out(_ptr(part_o), _ptr(part_ml), c_int(nsplit), c_int(H), c_int(K), c_int(V), _ptr(sink), _ptr(rows), c_int(nrows),
                              _ptr(uv), c_int(int(uv.dtype == torch.float32)), _ptr(out), c_int(out.stride(0)), _stream()), "pk_latent_out")


def latent_prefill(q: torch.Tensor, nrows: int, kv: torch.Tensor, kv_rows: int, tiles: torch.Tensor, ntiles: int, seqs: torch.Tensor,
                   gather: torch.Tensor, H: int, qk_panels: int, v_panels: int, V: int, window: int, scale: float, sink: torch.Tensor | None,
                   out: torch.Tensor, status: torch.Tensor) -> None:
    _check(_k().pk_latent_prefill(_ptr(q), c_int(nrows), _ptr(kv), c_int(kv_rows), _ptr(tiles), c_int(ntiles), _ptr(seqs), _ptr(gather), c_int(H),
                                  c_int(qk_panels), c_int(v_panels), c_int(V), c_int(window), c_float(scale), _ptr(sink), _ptr(out),
                                  c_int(out.stride(0)), _ptr(status), _stream()), "pk_latent_prefill")
