"""Operations of decoders with an fp32 residual stream.

RMS norms on the OUTPUT of each sublayer: ``embed_sinusoid`` starts the stream, ``stream_update`` adds a normalised
sublayer result (and hands out the stream as the next sublayer's operand in the same kernel).  RMS norms on the INPUT:
``stream_norms`` starts the stream or adds a result and hands out up to two normalised copies.  ``rms_rows`` is the norm
in front of the vocabulary projection, ``softcap`` limits the logits.  CUDA: csrc/kernels/residual_stream.cu; CPU tensors take an fp32 restatement.
"""
from __future__ import annotations

import ctypes
from ctypes import Structure, c_float, c_int32, c_int64, c_void_p

import torch

from . import _lib


class StreamUpdateArgs(Structure):
    """Mirror of ``cgk_stream_update_args`` (include/cogito_kernels.h)."""

    _fields_ = [("y", c_void_p), ("ldy", c_int64), ("pairs", c_void_p), ("ldp", c_int64), ("row_of", c_void_p), ("weight", c_void_p),
                ("w", c_void_p), ("x", c_void_p), ("h", c_void_p), ("rows", c_int32), ("D", c_int32), ("top", c_int32),
                ("pair_rows", c_int32), ("y_fp32", c_int32), ("pairs_fp32", c_int32), ("h_fp32", c_int32), ("eps", c_float)]


class StreamNormsArgs(Structure):
    """Mirror of ``cgk_stream_norms_args`` (include/cogito_kernels.h)."""

    _fields_ = [("ids", c_void_p), ("table", c_void_p), ("y", c_void_p), ("ldy", c_int64), ("w1", c_void_p), ("w2", c_void_p), ("x", c_void_p),
                ("h1", c_void_p), ("h2", c_void_p), ("rows", c_int32), ("D", c_int32), ("vocab", c_int32), ("table_fp32", c_int32),
                ("y_fp32", c_int32), ("h_fp32", c_int32), ("mult", c_float), ("eps", c_float)]


def sinusoid_frequencies(width: int, base: float = 10000.0, device=None) -> torch.Tensor:
    """fp64 [ceil(width / 2)]: pair i of a position vector turns by base^(-2i / width) per position."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / width).to(device)


def embed_sinusoid(ids, pos, table, scale: float = 1.0, freq=None):
    """ids [N] int64, pos [N] int32 -> (stream fp32 [N, D], operand copy in the table's type)."""
    N, D = ids.shape[0], table.shape[1]
    if not table.is_cuda:
        x = table[ids].float() * scale
        if freq is not None:
            angle = pos.double()[:, None] * freq[None]
            x = x + torch.stack([torch.sin(angle), torch.cos(angle)], -1).reshape(N, -1)[:, :D].float()
        return x, x.to(table.dtype)
    x = torch.empty(N, D, dtype=torch.float32, device=table.device)
    h = torch.empty(N, D, dtype=table.dtype, device=table.device)
    f32 = int(table.dtype == torch.float32)
    _lib.check(_lib.lib().cgk_embed_sinusoid(ids.data_ptr(), pos.data_ptr(), table.data_ptr(), f32, float(scale), _lib.ptr(freq), x.data_ptr(),
                                             h.data_ptr(), f32, N, D, table.shape[0], _lib.stream_ptr()), "cgk_embed_sinusoid")
    _lib.count_launch()
    return x, h


def stream_update(x, y, w, eps: float, dtype, pairs=None, row_of=None, weight=None):
    """x [N, D] fp32, in place: x += rms_norm(v) * w with
    v[t] = y[t] + sum_k weight[t, k] * (pairs[row_of[t, k]] if row_of[t, k] >= 0 else x[t]).
    Returns the new stream in ``dtype``."""
    if not x.is_cuda:
        v = y.float().clone() if y is not None else torch.zeros_like(x)
        if pairs is not None:
            for k in range(row_of.shape[1]):
                r = row_of[:, k].long()
                e = torch.where((r >= 0)[:, None], pairs[r.clamp_min(0)].float(), x)
                v = v + weight[:, k:k + 1] * e
        x += v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps) * w
        return x.to(dtype)
    N, D = x.shape
    h = torch.empty(N, D, dtype=dtype, device=x.device)
    a = StreamUpdateArgs()
    if y is not None:
        a.y, a.ldy, a.y_fp32 = y.data_ptr(), y.stride(0), int(y.dtype == torch.float32)
    if pairs is not None:
        a.pairs, a.ldp, a.pairs_fp32, a.pair_rows = pairs.data_ptr(), pairs.stride(0), int(pairs.dtype == torch.float32), pairs.shape[0]
        a.row_of, a.weight, a.top = row_of.data_ptr(), weight.data_ptr(), row_of.shape[1]
    a.w, a.x, a.h = w.data_ptr(), x.data_ptr(), h.data_ptr()
    a.rows, a.D, a.h_fp32, a.eps = N, D, int(dtype == torch.float32), float(eps)
    _lib.check(_lib.lib().cgk_stream_update(ctypes.byref(a), _lib.stream_ptr()), "cgk_stream_update")
    _lib.count_launch()
    return h


def stream_norms(x, eps: float, dtype, w1=None, w2=None, y=None, mult: float = 1.0, ids=None, table=None):
    """x [N, D] fp32, in place: x = table[ids], or x += mult * y, or unchanged.  Returns (h1, h2): the RMS-normed new
    stream times w1 and times w2 in ``dtype`` (None where the weight is None)."""
    if not x.is_cuda:
        if ids is not None:
            x.copy_(table[ids].float())
        elif y is not None:
            x += mult * y.float()
        n = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps)
        return tuple(None if w is None else (n * w).to(dtype) for w in (w1, w2))
    N, D = x.shape
    h = [None if w is None else torch.empty(N, D, dtype=dtype, device=x.device) for w in (w1, w2)]
    a = StreamNormsArgs()
    if ids is not None:
        a.ids, a.table, a.vocab, a.table_fp32 = ids.data_ptr(), table.data_ptr(), table.shape[0], int(table.dtype == torch.float32)
    if y is not None:
        a.y, a.ldy, a.y_fp32 = y.data_ptr(), y.stride(0), int(y.dtype == torch.float32)
    a.w1, a.w2, a.x, a.h1, a.h2 = _lib.ptr(w1), _lib.ptr(w2), x.data_ptr(), _lib.ptr(h[0]), _lib.ptr(h[1])
    a.rows, a.D, a.h_fp32, a.mult, a.eps = N, D, int(dtype == torch.float32), float(mult), float(eps)
    _lib.check(_lib.lib().cgk_stream_norms(ctypes.byref(a), _lib.stream_ptr()), "cgk_stream_norms")
    _lib.count_launch()
    return tuple(h)


def softcap(x, cap: float):
    """cap * tanh(x / cap), in place (fp32)."""
    if not x.is_cuda:
        return x.copy_(cap * torch.tanh(x / cap))
    if not x.is_contiguous():
        raise ValueError("softcap: contiguous logits expected")
    _lib.check(_lib.lib().cgk_softcap(x.data_ptr(), x.numel(), float(cap), _lib.stream_ptr()), "cgk_softcap")
    _lib.count_launch()
    return x


def rms_rows(x, w, eps: float, dtype, rows=None):
    """rms_norm(x[rows]) * w in ``dtype``; x fp32 [N, D], rows int64 or None for all."""
    if not x.is_cuda:
        v = x if rows is None else x[rows]
        return (v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps) * w).to(dtype)
    n = x.shape[0] if rows is None else rows.shape[0]
    out = torch.empty(n, x.shape[1], dtype=dtype, device=x.device)
    _lib.check(_lib.lib().cgk_rms_rows(x.data_ptr(), _lib.ptr(rows), n, x.shape[0], w.data_ptr(), out.data_ptr(), int(dtype == torch.float32),
                                       x.shape[1], float(eps), _lib.stream_ptr()), "cgk_rms_rows")
    _lib.count_launch()
    return out
