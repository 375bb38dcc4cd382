"""Recurrent mixers: linear attention whose state decays row by row (``ops.recurrence``).

``GatedLinearAttention``  keys of its own, decay sigmoid(W_a2 W_a1 h + b)^(1 / tau), result gated by silu(W_g h).
``Hgrn2``                 the forget gate f between a lower bound and 1 is the decay, and 1 - f the key.

Both RMS-norm every head's result with one weight.  They write the heads' results before the output product."""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..ops import recurrence as R
from ..ops.linear import linear
from .latent_attention import _frozen
from .parallel_layer import rows_of_8


@dataclass(frozen=True)
class RecurrentSpec:
    heads: int
    dim: int               # state rows per head
    vdim: int              # state columns per head
    tau: float = 1.0       # GatedLinearAttention: the decay's root


class _Recurrent(nn.Module):
    def __init__(self, spec: RecurrentSpec, tensors, device, dtype):
        super().__init__()
        self.spec = spec
        self._t = {k: v.to(device) for k, v in tensors.items()}
        # rows of a product start on 16 bytes: its columns are filled up to a multiple of 8
        self._put = lambda *names: _frozen(rows_of_8(torch.cat([self._t[n] for n in names], 0)).to(dtype).contiguous())
        self._vec = lambda name: _frozen(self._t[name].float().contiguous())

    def _loaded(self):
        del self._t, self._put, self._vec

    @property
    def out_width(self) -> int:
        return self.spec.heads * self.spec.vdim

    def _columns(self, x, *widths):
        at, out = 0, []
        for w in widths:
            out.append(x[:, at:at + w])
            at += w
        return out

    def forward(self, h: torch.Tensor, batch, cache, layer: int, out: torch.Tensor) -> torch.Tensor:
        """h [N, width], the tokens of ``batch``; writes to ``out`` [N, heads * vdim] and advances the layer's states in ``cache``."""
        return R.advance(self.rule, self.operands(h), cache.states[layer], batch, out)


class GatedLinearAttention(_Recurrent):
    """``tensors``: q, k, v, g, a1, a2 as [out, in] matrices, a2.b, norm."""

    def __init__(self, spec: RecurrentSpec, tensors, eps: float, device, dtype):
        super().__init__(spec, tensors, device, dtype)
        self.rule = R.StateRule(spec.heads, spec.dim, spec.vdim, R.ROOT, eps, q_scale=spec.dim ** -0.5, tau=spec.tau)
        self.w_in, self.w_a2 = self._put("q", "k", "v", "g", "a1"), self._put("a2")
        self.bias, self.norm = self._vec("a2.b"), self._vec("norm")
        self._loaded()

    def operands(self, h):
        s = self.spec
        x = linear(h, self.w_in, out_dtype=h.dtype)
        q, k, v, g, u = self._columns(x, s.heads * s.dim, s.heads * s.dim, s.heads * s.vdim, s.heads * s.vdim, self.w_a2.shape[1])
        z = linear(u, self.w_a2, out_dtype=torch.float32)[:, :s.heads * s.dim]
        return R.Operands(q, k, v, g, z, self.bias, None, self.norm)


class Hgrn2(_Recurrent):
    """``tensors``: q, f, v as [out, in] matrices, f.b, lower, norm."""

    def __init__(self, spec: RecurrentSpec, tensors, eps: float, device, dtype):
        super().__init__(spec, tensors, device, dtype)
        self.rule = R.StateRule(spec.heads, spec.dim, spec.vdim, R.BOUNDED, eps, q_silu=True)
        self.w_in, self.w_f = self._put("q", "v"), self._put("f")
        self.bias, self.low, self.norm = self._vec("f.b"), self._vec("lower"), self._vec("norm")
        self._loaded()

    def operands(self, h):
        s = self.spec
        q, v = self._columns(linear(h, self.w_in, out_dtype=h.dtype), s.heads * s.dim, s.heads * s.vdim)
        z = linear(h, self.w_f, out_dtype=torch.float32)[:, :s.heads * s.dim]
        return R.Operands(q, None, v, None, z, self.bias, self.low, self.norm)
