"""Projections of inference models: the tensor-core GEMM for many rows, a weight-streaming kernel
(csrc/kernels/skinny_gemm.cu) for up to ``FEW_ROWS`` (decoding).  fp32 operands and CPU tensors go through
``ops.gemm``."""
from __future__ import annotations

import torch

from . import _lib
from . import misc as M
from .gemm import _ld, gemm

FEW_ROWS = 8


def _few(a, b, mode_mn: bool) -> bool:
    if not a.is_cuda or a.dtype != torch.bfloat16 or a.shape[-2] > FEW_ROWS:
        return False
    ok = lambda t: t.stride(-1) == 1 and t.data_ptr() % 16 == 0 and all(s % 8 == 0 for s in t.stride()[:-1])
    return ok(b) and (b.shape[-1] % 8 == 0 if mode_mn else (a.shape[-1] % 8 == 0 and ok(a)))


def _skinny(a, b, out, mode: int, N: int):
    batch = a.shape[0] if a.dim() == 3 else 1
    s = [t.stride(0) if t.dim() == 3 else 0 for t in (a, b, out)]
    _lib.check(_lib.lib().cgk_skinny_gemm(a.data_ptr(), _ld(a), s[0], b.data_ptr(), _ld(b), s[1], out.data_ptr(), _ld(out), s[2],
                                          int(out.dtype == torch.float32), a.shape[-2], N, a.shape[-1], batch, mode, _lib.stream_ptr()),
               "cgk_skinny_gemm")
    _lib.count_launch()
    return out


def linear(a, w, *, w_mn: bool = False, out=None, out_dtype=torch.bfloat16):
    """a [.., M, K] times w [.., N, K] (or [.., K, N] with ``w_mn``), at most one batch dimension, strided views allowed."""
    if not _few(a, w, w_mn):
        return gemm(a, w, b_mn=w_mn, out=out, out_dtype=out_dtype)
    N = w.shape[-1] if w_mn else w.shape[-2]
    if out is None:
        out = torch.empty(*a.shape[:-1], N, dtype=out_dtype, device=a.device)
    return _skinny(a, w, out, 2 if w_mn else 0, N)


def gated_linear(a, w_gate_up, act: str = "silu", out=None):
    """act(a W_gate^T) * (a W_up^T); w_gate_up [2F, K]: gate rows, then up rows; act silu or relu; out may be a view
    with longer rows."""
    if not _few(a, w_gate_up, False):
        return M.gated(gemm(a, w_gate_up), act, out)
    F = w_gate_up.shape[0] // 2
    if out is None:
        out = torch.empty(a.shape[0], F, dtype=a.dtype, device=a.device)
    return _skinny(a, w_gate_up, out, 3 if act == "relu" else 1, F)
