"""Python faces of the sm_100a kernels (ctypes over ``libb200_cuda.so``).

Every function takes torch CUDA tensors, launches on the current torch stream and raises on a
non-zero return code.  There is no fallback: on a machine with a GPU a missing library is an error.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import c_double, c_float, c_int, c_long, c_size_t, c_void_p

import torch

from .. import _native

WT_Q4KR, WT_Q6KR, WT_Q8R, WT_BF16, WT_MXFP4R = 0, 1, 2, 3, 4
EPI_STORE, EPI_RESID, EPI_SWIGLU_Q8, EPI_SWIGLU_F32, EPI_ALLREDUCE, EPI_RELU2, EPI_GELU_ERF = 0, 1, 2, 3, 4, 6, 7
SYM_NONE, SYM_ALLREDUCE, SYM_RSCATTER, SYM_RSCATTER_ROWS = 0, 1, 2, 3
EMB_F32, EMB_BF16, EMB_Q8R, EMB_Q6KR = 0, 1, 2, 3
SCORE_SOFTMAX, SCORE_SIGMOID = 0, 1
ACT_NONE, ACT_GELU, ACT_SWIGLU_PAIR, ACT_RELU2, ACT_GELU_ERF = 0, 1, 2, 3, 4

_P = c_void_p
_DELTA = [_P, c_int, _P, c_int, _P, c_int] + [_P] * 8 + [c_int] * 5 + [c_float, c_float, _P, _P, c_int]
_SSD = [_P, c_int, c_int, c_int] + [_P] * 11 + [c_int] * 7 + [_P, c_int]
_SIGS = {
    "b200_embedding": [_P, _P, c_int, c_int, c_int, _P, _P, c_int, c_int, c_float, _P],
    "b200_rmsnorm": [_P, _P, c_float, c_int, c_int, _P, _P, _P, _P, _P, _P, c_int, _P, c_long, c_size_t, c_int, _P, _P],
    "b200_rmsnorm_allgather": [_P, _P, c_float, c_int, c_int, c_int, c_size_t, _P, _P],
    "b200_quantize_x": [_P, c_int, c_int, _P, _P, _P, _P],
    "b200_rope_kv": [_P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_float, _P, c_int, _P],
    "b200_rope_table": [_P, c_int, c_int, c_float, _P, _P],
    "b200_swiglu": [_P, c_int, c_int, _P, _P, c_int, _P],
    "b200_add_inplace": [_P, _P, c_size_t, _P],
    "b200_argmax": [_P, c_int, c_int, _P, _P, c_int, _P, _P],
    "b200_sample_topk": [_P, c_int, c_int, c_float, c_int, c_float, _P, _P, _P, _P],
    "b200_matvec_rope_kv": [c_int, _P, _P, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, _P, c_int, _P, _P, _P, c_int, c_int, c_int,
                            c_int, c_float, c_float, _P],
    "b200_matvec": [c_int, _P, _P, c_int, c_int, c_int, _P, _P, _P, _P, c_int, _P, _P, _P, c_int, _P, _P, _P, _P,
                    c_size_t, c_int, c_float, _P, _P],
    "b200_argmax_merge": [_P, _P, c_int, _P, c_size_t, c_int, _P],
    "b200_attn_decode": [_P, _P, _P, _P, c_int, c_int, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, _P, _P, _P,
                         _P, _P, _P, _P, _P, _P],
    "b200_attn_prefill": [_P, _P, _P, _P, c_int, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, _P],
    "b200_attn_prefill_tc05": [_P, _P, _P, _P, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P,
                               c_int, _P, c_int, c_int, _P, _P, _P],
    "b200_attn_prefill_latent": [_P, _P, c_long, c_int, c_int, _P, _P, c_int, c_int, c_int, _P, c_int, _P, _P, _P] + [c_int] * 7 + [_P, _P, c_int, _P, _P, _P],
    "b200_gemm_bf16": [_P, _P, c_int, c_int, c_int, c_int, c_int, _P, _P, c_int, _P, _P, _P, c_int, c_int, c_int, c_int,
                       _P, c_int, _P, c_size_t, c_int, c_int, c_int, c_int, c_int, c_float, c_int, _P, _P],
    "b200_gemm_heads": [_P, _P] + [c_int] * 7 + [_P, _P, c_int, c_int, c_float, _P, c_int, c_int, _P, _P],
    "b200_moe_gemm": [_P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, _P, c_int, _P, _P, _P, c_size_t, _P, c_long, _P, _P],
    "b200_moe_route_dispatch": [_P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_size_t, c_size_t, c_size_t, c_size_t,
                                _P, _P, c_int, c_float, _P, _P, _P],
    "b200_expert_gate_up": [_P, c_int, c_int, _P, c_int, _P, _P, c_int, _P, _P],
    "b200_expert_up": [_P, c_int, c_int, _P, c_int, _P, _P, c_int, _P, _P],
    "b200_expert_down": [_P, c_int, c_int, _P, c_int, _P, c_int, _P, _P, c_int, _P],
    "b200_depth_norm": [_P, c_size_t, _P, c_int, c_int, c_int, c_int, _P, _P, _P, _P, c_float, _P, _P, _P, _P, _P, c_long, _P, _P, _P, c_int, c_int, _P],
    "b200_poly_norm": [_P, c_int, c_int, c_int, c_int, _P, c_float, _P, _P, c_int, _P],
    "b200_mixed_finish": [_P] + [c_int] * 3 + [_P, _P, c_float, _P] + [c_int] * 5 + [_P, _P, _P, c_int, _P],
    "b200_mixed_decode": [_P] * 5 + [c_int, c_int, _P] + [c_int] * 6 + [_P] * 5,
    "b200_mixed_decode_prepare": [_P, _P, c_int, c_int, c_int, _P, _P],
    "b200_mixed_decode_ok": [c_int] * 3,
    "b200_mixed_prefill": [_P] * 5 + [c_int, _P, _P, _P] + [c_int] * 7 + [_P] * 4,
    "b200_mixed_prefill_ok": [c_int] * 2,
    "b200_moe_zero": [_P, c_int, _P],
    "b200_set_pdl": [c_int],
    "b200_set_prefetch": [c_int],
    "b200_dequant_bf16": [c_int, _P, _P, _P, c_size_t, c_int, _P],
    "b200_f32_to_bf16": [_P, _P, c_size_t, _P],
    "b200_transpose_bf16": [_P, _P, c_int, c_int, _P],
    "b200_qgemm": [c_int, _P, _P, c_int, c_int, _P, c_int, c_int, _P, _P, c_int, _P, c_int, c_int, _P, _P],
    "b200_decode_advance": [_P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P, _P, c_int, _P],
    "b200_modp_matvec": [_P, _P, _P, c_int, c_int, ctypes.c_uint, _P],
    "b200_modp_matmul": [_P, _P, _P, c_int, c_int, c_int, ctypes.c_uint, _P],
    "b200_count_mismatch": [_P, _P, c_size_t, _P, _P],
    "b200_norm_residual": [_P, c_int, _P, _P, c_int, c_int, _P, c_float, _P, _P, c_int, c_int, _P, c_long, _P, c_long, _P],
    "b200_qkv_finish": [_P, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, c_int, c_double, c_int, c_int, c_int, c_int, c_int, c_int,
                        c_int, c_int, c_int, c_float, c_float, c_int, _P, _P, _P, _P, c_int, c_int, c_int, _P, _P],
    "b200_attn_exact": [_P, _P, _P, c_int, _P, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, _P, _P, c_int, c_int, c_int,
                        c_int, _P, c_int, _P, c_int, _P],
    "b200_gemm_f32": [_P, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_float, c_int, _P, c_int, c_int, c_int, c_int, _P, _P],
    "b200_head_matvec": [_P, c_int, _P, c_int, _P] + [c_int] * 5 + [c_float, _P, c_int, c_int, c_int, _P],
    "b200_norm_dyt": [_P, c_int, c_int, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, _P, c_long, _P],
    "b200_diff_combine": [_P, _P, c_int, c_int, c_int, c_int, c_int, c_float, c_float, _P, _P, c_int, _P],
    "b200_latent_finish": [_P] + [c_int] * 10 + [_P, _P, c_float, _P, _P, _P, c_int, c_double, _P, _P, c_int, c_int, c_int, _P, c_int, _P],
    "b200_latent_q": [_P] + [c_int] * 12 + [_P, _P, c_int, c_double, c_float, _P, _P, _P],
    "b200_latent_gather": [_P, c_int, c_int, _P, c_int, _P, _P, c_int, c_int, _P, _P],
    "b200_latent_decode": [_P, _P, _P, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, c_int, _P, _P],
    "b200_latent_decode_ok": [c_int, c_int, c_int],
    "b200_logits_finish": [_P, c_size_t, c_float, c_float, _P],
    "b200_row_qkv_finish": [_P] + [c_int] * 5 + [_P] * 5 + [c_int] * 10 + [c_float, c_float, c_int] + [_P] * 6 + [c_int, _P],
    "b200_group_norm": [_P, c_int, _P, c_int, c_int, c_int, c_int, _P, c_float, _P, _P, c_int, _P],
    "b200_delta_recurrent": _DELTA + [_P],
    "b200_delta_chunked": _DELTA + [c_int, c_int, _P, c_size_t, _P],
    "b200_ssd_decode": _SSD + [_P, c_size_t, _P],
    "b200_ssd_prefill": _SSD + [c_int, c_int, c_int, _P, c_size_t, _P],
    "b200_gla_chunked": [_P] + [c_int] * 7 + [_P] * 8 + [c_int] * 5 + [c_float] * 3 + [_P, _P, c_int, c_int, c_int, _P, c_size_t, _P],
    "b200_gla_recurrent": [_P] + [c_int] * 7 + [_P] * 8 + [c_int] * 5 + [c_float] * 3 + [_P, _P, c_int, _P],
}

_lib = None


def lib():
    global _lib
    if _lib is None:
        L = _native.cuda()
        for name, args in _SIGS.items():
            if _native.cuda_subset and not hasattr(L, name):       # a partial library: kernels of other families are not in it
                continue
            fn = getattr(L, name)
            fn.argtypes = args
            fn.restype = c_int
        L.b200_attn_decode_scratch_floats.argtypes = [c_int, c_int, c_int, c_int, c_int]
        L.b200_attn_decode_scratch_floats.restype = c_size_t
        L.b200_latent_decode_scratch_floats.argtypes = [c_int] * 4
        L.b200_latent_decode_scratch_floats.restype = c_size_t
        L.b200_mixed_decode_scratch_floats.argtypes = [c_int] * 5
        L.b200_mixed_decode_scratch_floats.restype = c_size_t
        L.b200_mixed_decode_prepared_words.argtypes = [c_int] * 3
        L.b200_mixed_decode_prepared_words.restype = c_size_t
        L.b200_delta_chunk_bytes.argtypes = [c_int] * 5 + [c_float]
        L.b200_delta_chunk_bytes.restype = c_size_t
        L.b200_ssd_decode_bytes.argtypes = [c_int] * 5
        L.b200_ssd_decode_bytes.restype = c_size_t
        L.b200_ssd_prefill_bytes.argtypes = [c_int] * 7
        L.b200_ssd_prefill_bytes.restype = c_size_t
        L.b200_gla_chunk_bytes.argtypes = [c_int] * 6
        L.b200_gla_chunk_bytes.restype = c_size_t
        _lib = L
        if os.environ.get("B200_PDL", "1") == "0":      # debugging aid: fully serialised launches
            L.b200_set_pdl(0)
        if os.environ.get("B200_PREFETCH", "1") == "0":
            L.b200_set_prefetch(0)
    return _lib


def _p(t):
    return None if t is None else t.data_ptr()


def _sym(table):
    """ctypes pointer to a SymTable structure (or None)."""
    return None if table is None else ctypes.addressof(table)


def _st():
    return torch.cuda.current_stream().cuda_stream


def _check(rc: int, what: str):
    if rc != 0:
        raise RuntimeError(f"{what} failed with code {rc}")


def embedding(ids, out, emb_type, w, w2=None, vocab_lo=0, vocab_n=None, scale=1.0):
    T, D = out.shape
    _check(lib().b200_embedding(_p(ids), _p(out), T, D, emb_type, _p(w), _p(w2), vocab_lo,
                                vocab_n if vocab_n is not None else 2 ** 31 - 1, scale, _st()), "embedding")


def rmsnorm(x, g, eps, xq=None, xd=None, xs16=None, hb=None, hf=None, signal_sym=None, zero=None, slots=None):
    """``signal_sym``: symmetric-heap table; the kernel then ends by telling every rank that this rank has
    finished reading ``x`` (the handshake the fused all-reduce kernels check with ``wait_ready``).
    ``zero``: a contiguous fp32 tensor the kernel clears on the side (the output of a split-K GEMM that follows).
    ``slots``: ``(table, heap offset, rows, part)``: tensor parallel: ``part`` (fp32 [T, D], local) holds this rank's
    partial result of the row-parallel projection before this norm; the kernel all-reduces it through the per-rank slot
    tensor at ``heap offset`` ([2][world][rows][D] fp32 on every rank), adds the sum into ``x`` (in place), normalises
    it, and leaves ``part`` zeroed."""
    T, D = x.shape
    part = None
    if slots is not None:
        table, slot_off, slot_rows, part = slots
        mode = 2
    else:
        table, slot_off, slot_rows = signal_sym, 0, 0
        mode = 1 if signal_sym is not None else 0
    _check(lib().b200_rmsnorm(_p(x), _p(g), eps, T, D, _p(xq), _p(xd), _p(xs16), _p(hb), _p(hf), _sym(table), mode,
                              _p(zero), zero.numel() if zero is not None else 0, slot_off, slot_rows, _p(part), _st()), "rmsnorm")


def rmsnorm_allgather(x, g, eps, row0, n_rows, hb_off, sym):
    """Normalise rows [row0, row0 + n_rows) of ``x`` (fp32 [*, D]) and push them as bf16 into every rank's
    [*, D] tensor at byte offset ``hb_off`` of the symmetric heap; ends by bumping this rank's all-gather counter."""
    _check(lib().b200_rmsnorm_allgather(_p(x), _p(g), eps, row0, n_rows, x.shape[1], hb_off, _sym(sym), _st()), "rmsnorm_allgather")


def quantize_x(x, xq, xd, xs16):
    T, D = x.shape
    _check(lib().b200_quantize_x(_p(x), T, D, _p(xq), _p(xd), _p(xs16), _st()), "quantize_x")


def rope_kv(qkv, pos, slot, q_out, q_out_h, kc, vc, Hq, Hkv, hd, page_size, theta, style, q_scale, table=None):
    """``table``: optional (cos, sin) table from :func:`rope_table`; without it the angles are computed per call."""
    T = qkv.shape[0]
    _check(lib().b200_rope_kv(_p(qkv), _p(pos), _p(slot), _p(q_out), _p(q_out_h), _p(kc), _p(vc), T, Hq, Hkv, hd,
                              page_size, theta, style, q_scale, _p(table), 0 if table is None else table.shape[0], _st()),
           "rope_kv")


def rope_table(n_pos, hd, theta, device, freq=None):
    """fp32 [n_pos][hd/2][2] table of (cos, sin), computed in double precision on the device; ``freq``: hd/2 frequencies (numbers) in place of the
    powers of ``theta``."""
    tab = torch.empty((n_pos, hd // 2, 2), dtype=torch.float32, device=device)
    f = None if freq is None else torch.tensor(freq, dtype=torch.float64, device=device)
    _check(lib().b200_rope_table(_p(tab), n_pos, hd, theta, _p(f), _st()), "rope_table")
    return tab


def swiglu(gu, F, ob=None, of=None, zero_after=False):
    """``gu`` fp32 [T, 2F] holds (gate_i, up_i) in adjacent columns; writes silu(gate) * up; ``zero_after`` clears ``gu``."""
    T = gu.shape[0]
    _check(lib().b200_swiglu(_p(gu), T, F, _p(ob), _p(of), int(zero_after), _st()), "swiglu")


def add_inplace(x, y):
    _check(lib().b200_add_inplace(_p(x), _p(y), x.numel(), _st()), "add_inplace")


def argmax(logits, out_id, out_val=None, vocab_offset=0, scratch=None):
    T, V = logits.shape
    _check(lib().b200_argmax(_p(logits), T, V, _p(out_id), _p(out_val), vocab_offset, _p(scratch), _st()), "argmax")


def argmax_scratch(T, device):
    """Zeroed scratch that lets :func:`argmax` split each row over many blocks."""
    return torch.zeros(T * 4, dtype=torch.int32, device=device)


def sample_topk(logits, temperature, top_k, top_p, u, out_id, scratch):
    T, V = logits.shape
    _check(lib().b200_sample_topk(_p(logits), T, V, temperature, top_k, top_p, _p(u), _p(out_id), _p(scratch), _st()),
           "sample_topk")


def matvec(wt, w, w2, N, K, nb, xq=None, xd=None, xs16=None, xf=None, epi=EPI_STORE, bias=None, resid=None, y=None,
           ldy=0, oq=None, od=None, os16=None, sym=None, sym_off=0, wait_ready=False, alpha=1.0, col_scale=None):
    """Quantized mat-vec for 1..8 tokens (see ``matvec.cu``).  ``alpha`` (a number) and ``col_scale`` [N] multiply what EPI_RESID adds.  The SwiGLU epilogues read ``w`` as 2N rows interleaved
    (gate_0, up_0, gate_1, ...)."""
    _check(lib().b200_matvec(wt, _p(w), _p(w2), N, K, nb, _p(xq), _p(xd), _p(xs16), _p(xf), epi, _p(bias), _p(resid),
                             _p(y), ldy, _p(oq), _p(od), _p(os16), _sym(sym), sym_off, int(wait_ready), alpha, _p(col_scale), _st()), "matvec")


def matvec_rope_kv(w, nb, pos, slot, q_out, kc, vc, Hq, Hkv, hd, page_size, theta, q_scale, xq=None, xd=None, xs16=None, xf=None,
                   bias=None, table=None):
    """The fused QKV projection of ``nb`` <= 8 tokens with the rotary embedding (adjacent-pair layout) and the paged-cache
    write in its epilogue: replaces ``matvec(..., EPI_STORE)`` + ``rope_kv`` on the small-batch decode path.  ``w``: a
    ``QWeight`` with (Hq + 2 Hkv) * hd rows."""
    _check(lib().b200_matvec_rope_kv(w.wt, _p(w.main), _p(w.plane2), w.K, nb, _p(xq), _p(xd), _p(xs16), _p(xf), _p(bias), _p(pos),
                                     _p(slot), _p(table), 0 if table is None else table.shape[0], _p(q_out), _p(kc), _p(vc), Hq, Hkv,
                                     hd, page_size, theta, q_scale, _st()), "matvec_rope_kv")


def argmax_merge(out_id, out_val, nb, sym, merge_off, rows):
    """Merge per-shard arg-max results across tensor-parallel ranks in one kernel (see ``decode_ops.cu``)."""
    _check(lib().b200_argmax_merge(_p(out_id), _p(out_val), nb, _sym(sym), merge_off, rows, _st()), "argmax_merge")


def attn_decode_scratch_floats(B, Hq, Hkv, hd, S):
    return lib().b200_attn_decode_scratch_floats(B, Hq, Hkv, hd, S)


def attn_decode(q, kc, vc, page_table, seq_lens, B, Hq, Hkv, hd, window=0, S=1, sinks=None, out_f32=None, out_bf16=None,
                oq=None, od=None, os16=None, scratch=None, counters=None, status=None, dv=None, gate=None, chunk=0):
    """``chunk`` > 0: keys of the token's own chunk of that many positions only.  ``hd`` / ``dv``: query-key and value head sizes (``dv`` defaults to ``hd``); ``gate``: fp32 [B, >= Hq] view whose sigmoid scales
    each head's output."""
    _check(lib().b200_attn_decode(_p(q), _p(kc), _p(vc), _p(page_table), page_table.shape[1], kc.shape[0], _p(seq_lens), _p(sinks),
                                  B, Hq, Hkv, hd, hd if dv is None else dv, window, chunk, S, _p(gate), 0 if gate is None else gate.stride(0),
                                  _p(out_f32), _p(out_bf16), _p(oq), _p(od), _p(os16),
                                  _p(scratch), _p(counters), _p(status), _st()), "attn_decode")


def attn_prefill(q, kc, vc, page_table, max_pages, q_start, q_len, ctx_len, n_seqs, max_q_len, Hq, Hkv, hd, window=0,
                 sinks=None, out_bf16=None, out_f32=None, lse=None):
    _check(lib().b200_attn_prefill(_p(q), _p(kc), _p(vc), _p(page_table), max_pages, _p(q_start), _p(q_len),
                                   _p(ctx_len), _p(sinks), n_seqs, max_q_len, Hq, Hkv, hd, window, _p(out_bf16),
                                   _p(out_f32), _p(lse), _st()), "attn_prefill")


def attn_prefill_tc05(q16, kc, vc, page_table, q_start, q_len, ctx_len, n_seqs, max_q_len, Hq, Hkv, window=0, sinks=None,
                      out_bf16=None, status=None, dk=128, dv=128, gate=None, chunk=0, maps=1, out_f32=None):
    """``chunk`` > 0: keys of the query's own chunk only; ``maps`` 2: see :func:`qkv_finish`; ``out_f32`` instead of ``out_bf16``.  Prefill attention on tcgen05 (fp16 q / cache, bf16 out; ``dk`` 64..256 and ``dv`` 64 or 128, multiples of 64); ``gate``: fp32
    [T, >= Hq] view whose sigmoid scales each head's output.  See ``attn_prefill_tc05.cu``."""
    _check(lib().b200_attn_prefill_tc05(_p(q16), _p(kc), _p(vc), _p(page_table), page_table.shape[1], kc.shape[0], _p(q_start),
                                        _p(q_len), _p(ctx_len), n_seqs, max_q_len, q16.shape[0], Hq, Hkv, dk, dv, window, _p(sinks),
                                        _p(gate), 0 if gate is None else gate.stride(0), _p(out_bf16), chunk, maps, _p(out_f32), _p(status),
                                        _st()), "attn_prefill_tc05")


def attn_prefill_latent(q16, ws, v_col, base, cache, r_col, page_table, q_start, q_len, ctx_len, n_seqs, max_q, H, kn, rr, dv, out_bf16, sinks=None,
                        gate=None, status=None):
    """:func:`attn_prefill_tc05` over an expanded context: ``ws`` fp16 [rows, >= H * (kn + dv)] (own key parts, then values from ``v_col`` on; sequence b from
    row ``base[b]`` on), the shared key part in the columns from ``r_col`` of the paged latent ``cache`` [pages, 16, ks]; ``gate``: fp32 [T, >= H * dv]."""
    _check(lib().b200_attn_prefill_latent(_p(q16), _p(ws), ws.shape[0], ws.stride(0), v_col, _p(base), _p(cache), cache.shape[0], cache.shape[-1], r_col,
                                          _p(page_table), page_table.shape[1], _p(q_start), _p(q_len), _p(ctx_len), n_seqs, max_q, q16.shape[0], H, kn, rr, dv,
                                          _p(sinks), _p(gate), 0 if gate is None else gate.stride(0), _p(out_bf16), _p(status), _st()), "attn_prefill_latent")


def gemm_bf16(A, B, M, N, K, lda=None, ldb=None, out_f32=None, out_bf16=None, ldc=None, bias=None, resid_f32=None,
              resid_bf16=None, act=ACT_NONE, accumulate=False, tile_n=0, status=None, sym_mode=SYM_NONE, sym=None,
              sym_off=0, rows_per_rank=0, split_k=0, wait_ready=False, ag_rows_per_rank=0, ag_epoch=0, mn_major=False, alpha=1.0,
              out_f16=None, col_scale=None):
    """``alpha`` multiplies the product, ``col_scale`` [N] what is stored or added; ``out_f16`` instead of ``out_bf16``: stored as fp16.  D[M][N] = A[M][K] @ B[N][K]^T with fused epilogue (see ``gemm_tc05.cu``).  ``ag_rows_per_rank`` > 0: the rows
    of A are all-gathered by push (``rmsnorm_allgather``) and each tile waits for its owners' counter to reach ``ag_epoch``.
    ``mn_major``: the operands are given as A [K][M] and B [K][N] (row strides ``lda`` / ``ldb``), i.e. D = A^T B: the weight
    gradient dW = dy^T x straight from dy and x, without transposed copies."""
    _check(lib().b200_gemm_bf16(_p(A), _p(B), M, N, K, lda or (M if mn_major else K), ldb or (N if mn_major else K), _p(out_f32),
                                _p(out_bf16 if out_f16 is None else out_f16), ldc or N,
                                _p(bias), _p(resid_f32), _p(resid_bf16), act, int(accumulate), tile_n, split_k, _p(status),
                                sym_mode, _sym(sym), sym_off, rows_per_rank, int(wait_ready), ag_rows_per_rank, ag_epoch,
                                int(mn_major), alpha, int(out_f16 is not None), _p(col_scale), _st()), "gemm_bf16")


def gemm_heads(A, B, heads, N, K, head_k, out, head_ldc, alpha=1.0, gate=None, status=None):
    """One product per head on the tensor cores: ``out[:, z * head_ldc + n] = alpha * A[:, z * head_k: + K] @ B[z * N + n]`` (bf16 operands; fp32, bf16 or
    fp16 ``out``), times the sigmoid of ``gate`` (fp32, a column per output column)."""
    f32 = out.dtype == torch.float32
    _check(lib().b200_gemm_heads(_p(A), _p(B), A.shape[0], heads, N, K, A.stride(0), head_k, B.stride(0), _p(out) if f32 else None, None if f32 else _p(out),
                                 out.stride(0), head_ldc, alpha, _p(gate), 0 if gate is None else gate.stride(0), int(out.dtype == torch.float16),
                                 _p(status), _st()), "gemm_heads")


def set_pdl(on: bool):
    """Turn programmatic dependent launch of the decode-path kernels on or off (on by default)."""
    _check(lib().b200_set_pdl(int(on)), "set_pdl")


def dequant_bf16(wt, w, w2, out, N, K):
    _check(lib().b200_dequant_bf16(wt, _p(w), _p(w2), _p(out), N, K, _st()), "dequant_bf16")


def f32_to_bf16(x, y):
    _check(lib().b200_f32_to_bf16(_p(x), _p(y), x.numel(), _st()), "f32_to_bf16")


def transpose_bf16(x, out):
    R, C = x.shape
    _check(lib().b200_transpose_bf16(_p(x), _p(out), R, C, _st()), "transpose_bf16")


def decode_advance(ids, out_ids, pos, slot, seq_lens, page_table, page_size, B, hist, step_counter, hist_cap):
    _check(lib().b200_decode_advance(_p(ids), _p(out_ids), _p(pos), _p(slot), _p(seq_lens), _p(page_table),
                                     page_table.shape[1], page_size, B, _p(hist), _p(step_counter), hist_cap, _st()),
           "decode_advance")


QEPI_STORE, QEPI_ADD, QEPI_SWIGLU = 0, 1, 2


def qgemm(w, x_bf16, T, out_f32=None, out_bf16=None, ldo=None, bias=None, epi=QEPI_STORE, split_k=0, status=None):
    """out[T][N] (+)= x[T][K] @ dequant(W)[N][K]^T with the dequantization inside the tcgen05 pipeline
    (``qgemm_tc05.cu``).  ``w`` is a QWeight in Q4_K-R or Q6_K-R; its packed planes are read as they are.
    ``QEPI_SWIGLU``: rows of ``w`` are (gate, up) pairs, ``out_bf16`` gets N/2 columns."""
    wt = {WT_Q4KR: 0, WT_Q6KR: 1}[w.wt]
    _check(lib().b200_qgemm(wt, _p(w.main), _p(w.plane2), w.N, w.K, _p(x_bf16), x_bf16.stride(0), T, _p(out_f32), _p(out_bf16),
                            ldo if ldo is not None else w.N, _p(bias), epi, split_k, _p(status), _st()), "qgemm")


# ---------------------------------------------------------------- mixture of experts
def moe_route_dispatch(h_bf16, h_f32, router_w, router_b, top_k, E_local, C, recv_x_off, recv_meta_off, recv_w_off, counts_off,
                       sym, topk_ids=None, topk_w=None, status=None, score=SCORE_SOFTMAX, scale=1.0):
    """Router + top-k + weights (``score``: softmax over the chosen, which is also the softmax over all of them renormalised, or each one's sigmoid; times
    ``scale``) + expert-parallel dispatch of ``h_bf16`` [T][d] (see
    ``moe.cu``); the router (fp32 weights) reads ``h_f32`` when given.  ``sym`` None: one rank, the offsets are addresses."""
    T, d = (h_bf16 if h_bf16 is not None else h_f32).shape
    E = router_w.shape[0]
    _check(lib().b200_moe_route_dispatch(_p(h_bf16), _p(h_f32), _p(router_w), _p(router_b), T, d, E, top_k, E_local, C, recv_x_off,
                                         recv_meta_off, recv_w_off, counts_off, _p(topk_ids), _p(topk_w), score, scale, _sym(sym),
                                         _p(status), _st()), "moe_route_dispatch")


def moe_gemm(A, B, groups, group_rows, N, K, counts, mode, out_bf16=None, ldc=0, meta=None, gate_w=None, sym=None,
             sym_off=0, status=None, lda=None, ldb=None, col_scale=None, live_rows=0):
    """Grouped expert GEMM (see ``gemm_tc05.cu``): mode 1 = gate/up with fused SwiGLU, mode 3 = up with the square of relu, mode 2 = down
    projection fused with the weighted combine into the source ranks' residual streams.  Mode 1 with ``gate_w``: the weight multiplies
    the expert's input.  Mode 2 without ``sym``: ``sym_off`` is the address of the fp32 [tokens, ldc] destination; ``col_scale`` [N] multiplies
    what is added.  ``live_rows``: the most rows all groups hold together."""
    _check(lib().b200_moe_gemm(_p(A), _p(B), groups, group_rows, N, K, lda or K, ldb or K, _p(counts), mode, _p(out_bf16),
                               ldc, _p(meta), _p(gate_w), _sym(sym), sym_off, _p(col_scale), live_rows, _p(status), _st()), "moe_gemm")


def moe_choose(h, router_w, top_k, ids, w, score=SCORE_SOFTMAX, scale=1.0):
    """The choice alone: expert ids (int32) and weights (fp32), [T, top_k], of the rows ``h`` (bf16 or fp32)."""
    f32, E = h.dtype == torch.float32, router_w.shape[0]
    moe_route_dispatch(None if f32 else h, h if f32 else None, router_w, None, top_k, E, 0, 0, 0, 0, 0, None, topk_ids=ids, topk_w=w, score=score,
                       scale=scale)


def expert_gate_up(x, w13, F, ids, weights, mid):
    """``mid[t, s] = silu(w g) * (w u)`` for the chosen experts of fp32 rows ``x`` [T, K]; ``w13`` bf16 [E * 2 F, K], rows interleaved (gate, up); ``ids`` /
    ``weights`` [T, top] (None: weights of one)."""
    _check(lib().b200_expert_gate_up(_p(x), x.shape[0], x.shape[1], _p(w13), F, _p(ids), _p(weights), ids.shape[1], _p(mid), _st()), "expert_gate_up")


def expert_up(x, w1, F, ids, weights, mid):
    """``mid[t, s] = w relu(u)^2`` for the chosen experts (no gate) of fp32 rows ``x`` [T, K]; ``w1`` bf16 [E * F, K]."""
    _check(lib().b200_expert_up(_p(x), x.shape[0], x.shape[1], _p(w1), F, _p(ids), _p(weights), ids.shape[1], _p(mid), _st()), "expert_up")


def expert_down(mid, w2, N, ids, out, scale=None):
    """``out[t] += scale * sum_s W_down[ids[t, s]] mid[t, s]``; ``w2`` bf16 [E * N, F]."""
    T, top = ids.shape
    _check(lib().b200_expert_down(_p(mid), T, w2.shape[1], _p(w2), N, _p(ids), top, _p(scale), _p(out), out.stride(0), _st()), "expert_down")


def moe_zero(t):
    _check(lib().b200_moe_zero(_p(t), t.numel(), _st()), "moe_zero")


# ---- exact arithmetic over a prime field (training verification): residues are int32 tensors with values in [0, p), p < 2^31
def modp_matvec(A, x, p: int):
    rows, cols = A.shape
    y = torch.empty(rows, dtype=torch.int32, device=A.device)
    _check(lib().b200_modp_matvec(_p(A), _p(x), _p(y), rows, cols, p, _st()), "modp_matvec")
    return y


def modp_matmul(A, B, p: int):
    n, k = A.shape
    m = B.shape[1]
    C = torch.empty((n, m), dtype=torch.int32, device=A.device)
    _check(lib().b200_modp_matmul(_p(A), _p(B), _p(C), n, k, m, p, _st()), "modp_matmul")
    return C


def count_mismatch(a, b) -> torch.Tensor:
    out = torch.zeros(1, dtype=torch.int32, device=a.device)
    _check(lib().b200_count_mismatch(_p(a), _p(b), a.numel(), _p(out), _st()), "count_mismatch")
    return out


# ---------------------------------------------------------------- hybrid stacks (attention and recurrent layers, norms on both sides)
def norm_residual(x, eps, y=None, gy=None, gh=None, hb=None, hf=None, y_clear=False, zero=None, zero2=None):
    """``x += y / rms(y) * gy`` (with ``y``), then ``h = x / rms(x) * gh`` (without ``gh``: ``h = x``) into ``hb`` (bf16) and/or ``hf`` (fp32), whose
    columns beyond x's width are written as zeros.  ``y_clear`` leaves y's rows zeroed; ``zero`` / ``zero2``: contiguous fp32
    tensors cleared on the side."""
    T, D = x.shape
    h = hb if hb is not None else hf
    _check(lib().b200_norm_residual(_p(y), 0 if y is None else y.stride(0), _p(gy), _p(x), T, D, _p(gh), eps, _p(hb), _p(hf),
                                    0 if h is None else h.stride(0), int(y_clear), _p(zero), 0 if zero is None else zero.numel(),
                                    _p(zero2), 0 if zero2 is None else zero2.numel(), _st()), "norm_residual")


def qkv_finish(proj, q_off, k_off, v_off, pos, slot, table, base, H, G, dim, vdim, DK, DV, rot, style, qk_norm, eps, q_scale, page_size,
               q32=None, q16=None, kc=None, vc=None, maps=1, q_wide=False, bias=None):
    """``bias`` is added to the projection row; ``maps`` 2 (differential attention): ``H`` counts the query rows of both maps, ordered (key/value head, map,
    head of the group), a cache row holds both maps' keys side by side, and ``q_wide`` pads a query with zeros on the other map's half.  Rotation, unit-RMS norm and scale of the queries and keys of a fused projection row, and the paged-cache write of keys and
    values (``k_off`` < 0: the layer has none); see ``hybrid_ops.cu``."""
    f32 = int(kc is not None and kc.dtype == torch.float32)
    _check(lib().b200_qkv_finish(_p(proj), proj.stride(0), proj.shape[0], q_off, k_off, v_off, _p(pos), _p(slot), _p(table),
                                 0 if table is None else table.shape[0], base, H, G, dim, vdim, DK, DV, rot, style, int(qk_norm), eps,
                                 q_scale, page_size, _p(q32), _p(q16), _p(kc), _p(vc), f32, maps, int(q_wide), _p(bias), _st()), "qkv_finish")


def attn_exact(q32, kc, vc, page_table, q_start, q_len, ctx_len, n_seqs, max_q, H, G, DK, DV, gate=None, out_f32=None, out_bf16=None, maps=1,
               chunk=0, sinks=None, window=0, slopes=None, slices=1):
    """Causal attention in 32-bit arithmetic for any head sizes; ``gate``: fp32 [T, >= H] view whose sigmoid scales each head; ``maps``: see
    :func:`qkv_finish`; ``vc`` None: the values are the first DV columns of the keys (latent attention); ``slopes`` [H]: times the distance, taken off
    the scores; ``slices``: see :func:`mixed_finish`."""
    o = out_f32 if out_f32 is not None else out_bf16
    _check(lib().b200_attn_exact(_p(q32), _p(kc), _p(vc), int(kc.dtype == torch.float32), _p(page_table), page_table.shape[1], _p(q_start),
                                 _p(q_len), _p(ctx_len), n_seqs, max_q, H, G, DK, DV, _p(gate), 0 if gate is None else gate.stride(0),
                                 _p(out_f32), _p(out_bf16), o.stride(0), kc.shape[-1], maps, chunk, _p(sinks), window, _p(slopes), slices, _st()), "attn_exact")


def gemm_f32(A, W, out, act=0, alpha=1.0, accumulate=False, gate=None, heads=1, head_k=0, head_ldc=0, col_scale=None):
    """``out = act(alpha * A @ W^T)`` in true 32-bit: A fp32 [M, K], W bf16 [N, K]; ``act`` 1: the square of relu, 2: the erf gelu; times the sigmoid of ``gate``
    [M, N] and by ``col_scale`` [N]; ``accumulate`` adds into ``out``.  ``heads`` > 1: one product per head, as in :func:`gemm_heads`."""
    M, (N, K) = A.shape[0], W.shape
    _check(lib().b200_gemm_f32(_p(A), A.stride(0), _p(W), W.stride(0), _p(out), out.stride(0), M, N // heads, K, act, alpha, int(accumulate), _p(gate),
                               0 if gate is None else gate.stride(0), heads, head_k, head_ldc, _p(col_scale), _st()), "gemm_f32")


def head_matvec(A, W, out, heads, head_k, head_ldc, alpha=1.0, gate=None):
    """:func:`gemm_heads` for 1..8 fp32 rows on the CUDA cores: ``W`` bf16 [heads * N, K]."""
    _check(lib().b200_head_matvec(_p(A), A.stride(0), _p(W), W.stride(0), _p(out), out.stride(0), A.shape[0], heads, W.shape[0] // heads, W.shape[1], alpha,
                                  _p(gate), 0 if gate is None else gate.stride(0), head_k, head_ldc, _st()), "head_matvec")


def depth_norm(xs, D, eps=0.0, weights=None, out=None, add=None, g1=None, g2=None, h1=None, h2=None, zero=None, base=None, parts=None,
               part_weights=None):
    """``x = sum_j weights[j] * xs[j]`` over the slabs of ``xs`` (fp32 [n, >= T, ld], D columns live; a slice along the rows is fine; ``weights`` None: one
    slab as it is); ``out`` [T, ld] = x + ``add``; ``h1`` / ``h2`` (both bf16 or fp32, [T, ld]) = x over its root mean square, times ``g1`` / ``g2``.
    ``base`` [T, ld] is added to x; ``parts`` [k, T, ld] (at most 3, slabs as far apart as those of ``xs``) take other weighted sums of the same slabs,
    ``part_weights`` [k, >= n]."""
    n, T, ld = xs.shape
    f32 = next((h.dtype == torch.float32 for h in (h1, h2) if h is not None), False)
    b, f = (lambda h: None if f32 else _p(h)), (lambda h: _p(h) if f32 else None)                   # noqa: E731
    _check(lib().b200_depth_norm(_p(xs), xs.stride(0), _p(weights), n, T, D, ld, _p(out), _p(add), _p(g1), _p(g2), eps, b(h1), b(h2), f(h1), f(h2),
                                 _p(zero), 0 if zero is None else zero.numel(), _p(base), _p(parts), _p(part_weights), 0 if parts is None else parts.shape[0],
                                 0 if parts is None else part_weights.stride(0), _st()), "depth_norm")
    assert parts is None or parts.stride(0) == xs.stride(0)


def poly_norm(z, F, coef, eps, out):
    """``a N(z) + b N(z^2) + c N(z^3) + e`` per row of ``z`` (fp32 or bf16 [T, >= F]), N dividing by the root mean square, ``coef`` = (a, b, c, e); ``out`` bf16 or fp32,
    columns beyond F zero."""
    f32 = out.dtype == torch.float32
    _check(lib().b200_poly_norm(_p(z), int(z.dtype == torch.bfloat16), z.stride(0), z.shape[0], F, _p(coef), eps, None if f32 else _p(out), _p(out) if f32 else None, out.stride(0), _st()),
           "poly_norm")


def mixed_finish(proj, k_off, bias, mix, scale, slot, H, G, dim, DK, q, kc):
    """Queries and keys of an attention layer whose heads' scores are mixed: a cache row holds all G heads' keys of DK columns side by side (they are the
    values too), and a query row ``q`` (fp32 or fp16 [T, H, G * DK]) holds, per key head, the ``mix`` [H, H] weighted sum of that group's scaled
    queries, so that its product with a cache row is the mixed score.  ``proj`` fp32 [T, >= (H + G) * dim], keys from column ``k_off`` on."""
    f32, c32 = q.dtype == torch.float32, kc.dtype == torch.float32
    _check(lib().b200_mixed_finish(_p(proj), proj.stride(0), proj.shape[0], k_off, _p(bias), _p(mix), scale, _p(slot), H, G, dim, DK, kc.shape[2],
                                   _p(q) if f32 else None, None if f32 else _p(q), _p(kc), int(c32), _st()), "mixed_finish")


def mixed_decode_ok(H, G, DK):
    return bool(lib().b200_mixed_decode_ok(H, G, DK))


def mixed_prefill_ok(G, DK):
    return bool(lib().b200_mixed_prefill_ok(G, DK))


def mixed_decode_scratch_floats(B, H, G, DK, S):
    return lib().b200_mixed_decode_scratch_floats(B, H, G, DK, S)


def mixed_decode_prepare(mix, slopes, H, G, DK):
    """The mixture (fp32 [H, H] of bf16 values) and the mixed scores' ``slopes`` [H] in the form :func:`mixed_decode` reads: once per layer, at load."""
    out = torch.empty(lib().b200_mixed_decode_prepared_words(H, G, DK), dtype=torch.int32, device=mix.device)
    _check(lib().b200_mixed_decode_prepare(_p(mix), _p(slopes), H, G, DK, _p(out), _st()), "mixed_decode_prepare")
    return out


def mixed_decode(q, kc, mix, page_table, seq_lens, B, H, G, DK, window=0, S=1, sinks=None, out_f32=None, out_bf16=None, scratch=None, status=None):
    """One query token per sequence, heads mixed on the scores (see ``mixed_attn.cu``): ``q`` fp32 [B, H, DK], scaled and not mixed; ``kc`` fp16 [pages, 1, 16,
    G * DK], keys and values; ``mix`` from :func:`mixed_decode_prepare`.  ``S``: shares of the keys, at most 64."""
    _check(lib().b200_mixed_decode(_p(q), _p(kc), _p(mix), _p(sinks), _p(page_table), page_table.shape[1], kc.shape[0], _p(seq_lens), B, H, G, DK,
                                   window, S, _p(out_f32), _p(out_bf16), _p(scratch), _p(status), _st()), "mixed_decode")


def mixed_prefill(q16, kc, slopes, page_table, q_start, q_len, ctx_len, n_seqs, max_q, H, G, DK, window=0, sinks=None, out_bf16=None, out_f32=None, status=None):
    """Prompt portions with wide queries: ``q16`` fp16 [T, H * G * DK] from :func:`mixed_finish`, against the same cache rows."""
    _check(lib().b200_mixed_prefill(_p(q16), _p(kc), _p(slopes), _p(sinks), _p(page_table), page_table.shape[1], _p(q_start), _p(q_len), _p(ctx_len),
                                    n_seqs, max_q, q16.shape[0], H, G, DK, window, _p(out_bf16), _p(out_f32), _p(status), _st()), "mixed_prefill")


def norm_dyt(x, alpha, w, b, hb=None, hf=None, ids=None, emb=None, zero=None):
    """``h = tanh(alpha * x) * w + b`` (Dynamic Tanh) into ``hb`` (bf16) and/or ``hf`` (fp32), padding columns zero; with ``emb`` (bf16 [vocab, D]) the
    tokens' rows of it are added to ``x`` first; ``zero``: a contiguous fp32 tensor cleared on the side."""
    T, D = x.shape
    h = hb if hb is not None else hf
    _check(lib().b200_norm_dyt(_p(x), T, D, _p(ids), _p(emb), 0 if emb is None else emb.shape[0], _p(alpha), _p(w), _p(b), _p(hb), _p(hf), h.stride(0),
                               _p(zero), 0 if zero is None else zero.numel(), _st()), "norm_dyt")


def diff_combine(maps_out, lam, H, G, vdim, DV, eps, mult, out_f32=None, out_bf16=None):
    """``o = a1 - lam * a2`` over two maps' outputs (fp32 [T, 2 H DV], :func:`qkv_finish`'s order), divided by its root mean square per head, times ``mult``."""
    o = out_f32 if out_f32 is not None else out_bf16
    _check(lib().b200_diff_combine(_p(maps_out), _p(lam), maps_out.shape[0], H, G, vdim, DV, eps, mult, _p(out_f32), _p(out_bf16), o.stride(0), _st()),
           "diff_combine")


# ---------------------------------------------------------------- latent attention (see ``latent_attn.cu``)
def latent_finish(proj, q_off, c_off, r_off, q_rank, rank, rot_dim, rot, style, q_w, c_w, eps, pos, slot, table, base, cq, cache, CR, RR):
    """RMS norm of the two latents of a down-projection row and rotation of the shared key part: the query latent to ``cq`` (bf16 or fp32, padded), the
    rest to the token's row of the paged ``cache`` [pages, 16, CR + RR]."""
    f32 = cq.dtype == torch.float32
    _check(lib().b200_latent_finish(_p(proj), proj.stride(0), proj.shape[0], q_off, c_off, r_off, q_rank, rank, rot_dim, rot, style, _p(q_w), _p(c_w), eps,
                                    _p(pos), _p(slot), _p(table), 0 if table is None else table.shape[0], base, _p(cq) if f32 else None,
                                    None if f32 else _p(cq), cq.stride(0), CR, RR, _p(cache), int(cache.dtype == torch.float32), _st()), "latent_finish")


def latent_q(q, hs, H, dim, rot_dim, rot, style, NC, r_col, RR, width, pos, table, base, scale, out):
    """Rotation and scale of the queries (fp32 [T, H * hs]) into ``out`` (fp32 or fp16 [T, H, width]): the unrotated part to columns [0, NC) (0: left alone),
    the rotated one to [r_col, r_col + RR)."""
    f32 = out.dtype == torch.float32
    _check(lib().b200_latent_q(_p(q), q.stride(0), hs, q.shape[0], H, dim, rot_dim, rot, style, NC, r_col, RR, width, _p(pos), _p(table),
                               0 if table is None else table.shape[0], base, scale, _p(out) if f32 else None, None if f32 else _p(out), _st()), "latent_q")


def latent_gather(cache, CR, page_table, ctx_len, base, n_seqs, max_ctx, out):
    """The cached latents (fp16) of whole contexts as rows of ``out`` (bf16 [rows, CR]), sequence b from row ``base[b]`` on."""
    _check(lib().b200_latent_gather(_p(cache), cache.shape[-1], CR, _p(page_table), page_table.shape[1], _p(ctx_len), _p(base), n_seqs, max_ctx, _p(out),
                                    _st()), "latent_gather")


def latent_decode_ok(H, CR, RR):
    return bool(lib().b200_latent_decode_ok(H, CR, RR))


def latent_decode_scratch_floats(R, H, CR, S):
    return lib().b200_latent_decode_scratch_floats(R, H, CR, S)


def latent_decode(q, cache, page_table, row_seq, pos, R, H, CR, RR, S, scratch, out_f32=None, out_bf16=None, sinks=None, status=None):
    """Attention of R query rows in the latent space: ``q`` fp32 [R, H, CR + RR] against the paged rows of ``cache``, as keys and as values; row r belongs to
    sequence ``row_seq[r]`` (None: r) and sees positions 0..``pos[r]``.  ``S``: shares of the keys."""
    o = out_f32 if out_f32 is not None else out_bf16
    _check(lib().b200_latent_decode(_p(q), _p(cache), _p(page_table), page_table.shape[1], cache.shape[0], _p(row_seq), _p(pos), _p(sinks), R, H, CR, RR, S,
                                    _p(scratch), _p(out_f32), _p(out_bf16), o.stride(0), _p(status), _st()), "latent_decode")


def logits_finish(logits, scale, cap):
    _check(lib().b200_logits_finish(_p(logits), logits.numel(), scale, cap, _st()), "logits_finish")


def gla_recurrent(proj, offs, rank, a2, b2, w, state, q_start, q_len, ctx_len, slots, n_seqs, H, dim, vdim, VP, tau, q_scale, eps,
                  out_f32=None, out_bf16=None):
    """Gated linear attention token by token over every sequence's new tokens (see ``linear_attn.cu``).  ``offs``: columns of q, k, v,
    the output gate and the low-rank decay input in ``proj``; ``a2`` fp32 [rank, H * dim]; ``state`` fp32 [slots, H, dim, VP]."""
    o = out_f32 if out_f32 is not None else out_bf16
    _check(lib().b200_gla_recurrent(_p(proj), proj.stride(0), *offs, rank, _p(a2), _p(b2), _p(w), _p(state), _p(q_start), _p(q_len),
                                    _p(ctx_len), _p(slots), n_seqs, H, dim, vdim, VP, tau, q_scale, eps, _p(out_f32), _p(out_bf16),
                                    o.stride(0), _st()), "gla_recurrent")


def gla_chunk_bytes(T, n_seqs, H, dim, VP, rank):
    """Workspace of :func:`gla_chunked`; 0 for sizes it does not take."""
    return lib().b200_gla_chunk_bytes(T, n_seqs, H, dim, VP, rank)


def gla_chunked(proj, offs, rank, a2, b2, w, state, q_start, q_len, ctx_len, slots, n_seqs, H, dim, vdim, VP, tau, q_scale, eps, max_q, ws,
                out_f32=None, out_bf16=None):
    """:func:`gla_recurrent` for prompts, in 64-token chunks on the tensor cores; ``ws``: uint8 workspace."""
    o = out_f32 if out_f32 is not None else out_bf16
    _check(lib().b200_gla_chunked(_p(proj), proj.stride(0), *offs, rank, _p(a2), _p(b2), _p(w), _p(state), _p(q_start), _p(q_len),
                                  _p(ctx_len), _p(slots), n_seqs, H, dim, vdim, VP, tau, q_scale, eps, _p(out_f32), _p(out_bf16),
                                  o.stride(0), proj.shape[0], max_q, _p(ws), ws.numel(), _st()), "gla_chunked")


# ---------------------------------------------------------------- projections normed as whole rows, gated norm in parts
def row_qkv_finish(proj, q_off, k_off, v_off, q_w, k_w, pos, slot, table, H, G, dim, vdim, DK, DV, rot, style, v_norm, eps, q_scale, page_size, kc, vc,
                   q32=None, q16=None, lam=None, v_first=None):
    """Queries and keys of a fused projection row, each normed over all its heads together (``q_w`` / ``k_w``: weights per column, None: not normed), rotated and
    scaled; values normed per head (``v_norm``) and mixed, ``(1 - lam) v + lam v_first`` (without ``lam``: written to ``v_first``, fp32 [T, G * vdim], where
    given); keys and values to the paged cache."""
    _check(lib().b200_row_qkv_finish(_p(proj), proj.stride(0), proj.shape[0], q_off, k_off, v_off, _p(q_w), _p(k_w), _p(pos), _p(slot), _p(table),
                                     0 if table is None else table.shape[0], H, G, dim, vdim, DK, DV, rot, style, int(v_norm), eps, q_scale, page_size,
                                     _p(lam), _p(v_first), _p(q32), _p(q16), _p(kc), _p(vc), int(kc.dtype == torch.float32), _st()), "row_qkv_finish")


def group_norm(y, D, groups, w, eps, out, gate=None):
    """``v = y * silu(gate)`` (fp32 [T, >= D] views; ``gate`` None: ``v = y``), each of ``groups`` equal parts divided by its own root mean square, times ``w`` [D];
    ``out`` bf16 or fp32, columns beyond D zero."""
    f32 = out.dtype == torch.float32
    _check(lib().b200_group_norm(_p(y), y.stride(0), _p(gate), 0 if gate is None else gate.stride(0), y.shape[0], D, groups, _p(w), eps,
                                 None if f32 else _p(out), _p(out) if f32 else None, out.stride(0), _st()), "group_norm")


# ---------------------------------------------------------------- generalized delta rule (see ``delta_rule.cu``)
def _delta_args(proj, offs, rank, w2, w0, ab, norm, state, q_start, q_len, ctx_len, slots, n_seqs, H, dim, vdim, VP, decay, eps, out):
    f32 = out.dtype == torch.float32
    return (_p(proj), proj.stride(0), (c_int * 6)(*offs), rank, _p(w2), w2.shape[1], _p(w0), _p(ab), _p(norm), _p(state), _p(q_start), _p(q_len), _p(ctx_len),
            _p(slots), n_seqs, H, dim, vdim, VP, decay, eps, _p(out) if f32 else None, None if f32 else _p(out), out.stride(0))


def delta_recurrent(*args):
    """Generalized delta rule token by token over every sequence's new tokens.  Arguments: the fused projections; ``offs``: their columns of r, k, v, the output
    gate, the removal rate and the low-rank decay input; ``rank``; ``w2`` bf16 [H * dim, rank padded to 8]; ``w0`` and ``ab`` [H * dim]; ``norm`` [H * vdim];
    ``state`` fp32 [slots, H, dim, VP]; q_start, q_len, ctx_len, slots; n_seqs, H, dim, vdim, VP; ``decay`` (log w = -decay * sigmoid); eps; ``out`` (bf16 or
    fp32 [T, H * VP])."""
    _check(lib().b200_delta_recurrent(*_delta_args(*args), _st()), "delta_recurrent")


def delta_chunk_bytes(T, n_seqs, H, dim, VP, decay):
    """Workspace of :func:`delta_chunked`; 0 for sizes it does not take."""
    return lib().b200_delta_chunk_bytes(T, n_seqs, H, dim, VP, decay)


def delta_chunked(*args, max_q, ws):
    """:func:`delta_recurrent` for prompts, in 64-token chunks on the tensor cores; ``ws``: uint8 workspace."""
    _check(lib().b200_delta_chunked(*_delta_args(*args), args[0].shape[0], max_q, _p(ws), ws.numel(), _st()), "delta_chunked")


# ---------------------------------------------------------------- state-space duality (see ``ssd.cu``)
def _ssd_args(proj, x_off, dt_off, conv, conv_b, dt_bias, A_log, D, state, ring, q_start, q_len, ctx_len, slots, n_seqs, H, P, N, G, PP, y):
    return (_p(proj), proj.stride(0), x_off, dt_off, _p(conv), _p(conv_b), _p(dt_bias), _p(A_log), _p(D), _p(state), _p(ring), _p(q_start), _p(q_len), _p(ctx_len),
            _p(slots), n_seqs, H, P, N, G, conv.shape[1], PP, _p(y), y.stride(0))


def ssd_decode_bytes(n_seqs, H, PP, N, G):
    """Workspace of :func:`ssd_decode`."""
    return lib().b200_ssd_decode_bytes(n_seqs, H, PP, N, G)


def ssd_decode(*args, ws):
    """One token per sequence of a Mamba-2 layer: filter, recurrence and skip.  Arguments: the projections (fp32), their columns of [x, B, C] and of dt; ``conv`` fp32
    [channels, taps] and its bias; dt_bias, A_log, D [H]; ``state`` fp32 [slots, H, N, PP]; ``ring`` fp32 [slots, taps, channels]; q_start, q_len, ctx_len,
    slots; n_seqs, H, P, N, G, PP; ``y`` fp32 [T, >= H * P]; ``ws``: uint8 workspace."""
    _check(lib().b200_ssd_decode(*_ssd_args(*args), _p(ws), ws.numel(), _st()), "ssd_decode")


def ssd_prefill_bytes(T, n_seqs, H, PP, N, G, exact=False):
    return lib().b200_ssd_prefill_bytes(T, n_seqs, H, PP, N, G, int(exact))


def ssd_prefill(*args, max_q, ws, exact=False):
    """The same for prompts: 64-token chunks on the tensor cores, or (``exact``) token by token in fp32; ``ws``: uint8 workspace."""
    _check(lib().b200_ssd_prefill(*_ssd_args(*args), args[0].shape[0], max_q, int(exact), _p(ws), ws.numel(), _st()), "ssd_prefill")
