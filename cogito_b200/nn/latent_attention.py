"""Latent attention: queries and keys/values go through short RMS-normed vectors, and only the key/value latent
is cached.

    c_q = rms(W_dq h),  q = W_uq c_q            c = rms(W_dkv h),  k = W_uk c,  v = W_uv c     (per head)
    o = softmax(scale q k^T) v over the positions up to the query's own,   result W_o o

Two forms of the same sum.  Prompt portions expand k and v for the whole context with one product and use the
flash-attention kernel.  Single tokens and short portions stay in the latent space: q' = W_uk^T q meets the cached
latents directly and W_uv is applied to the result, so a step reads ``kv_rank`` numbers per cached token for all
heads together.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..ops.attention import flash_forward
from ..ops.linear import linear


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int               # query / key elements per head
    vdim: int              # value elements per head
    q_rank: int
    kv_rank: int
    scale: float           # of the scores


def _frozen(t: torch.Tensor) -> nn.Parameter:
    return nn.Parameter(t, requires_grad=False)


def _pad_heads(w: torch.Tensor, heads: int, dim: int, to: int) -> torch.Tensor:
    """[heads * dim, K] -> [heads * to, K] with zero rows after each head's own."""
    if dim == to:
        return w
    out = torch.zeros(heads, to, w.shape[1], dtype=w.dtype, device=w.device)
    out[:, :dim] = w.view(heads, dim, -1)
    return out.view(heads * to, -1)


class LatentAttention(nn.Module):
    """Inference module.  ``tensors``: dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o as [out, in] matrices and norm weights."""

    PROMPT_MIN = 32          # portions of at least this many tokens take the prompt form

    def __init__(self, spec: LatentSpec, tensors: dict[str, torch.Tensor], eps: float, device, dtype):
        super().__init__()
        self.spec, self.eps = spec, eps
        H = spec.heads
        t = {k: v.to(device) for k, v in tensors.items()}
        wide = max(spec.dim, spec.vdim)
        # The flash kernel takes heads of 64 or 128 elements: smaller ones get zero columns (exact).  Longer heads, and
        # fp32, use the latent form throughout.
        self.prompt_form = dtype == torch.bfloat16 and wide <= 128
        self.dq = self.dv = 64 if wide <= 64 else 128
        if not self.prompt_form:
            self.dq, self.dv = spec.dim, spec.vdim
        put = lambda w: _frozen(w.to(dtype).contiguous())
        self.w_down = put(torch.cat([t["dq"], t["dkv"]], 0))
        self.q_norm, self.kv_norm = _frozen(t["dq.norm"].float().contiguous()), _frozen(t["dkv.norm"].float().contiguous())
        self.w_uq = put(_pad_heads(t["uq"], H, spec.dim, self.dq))
        uk, uv = _pad_heads(t["uk"], H, spec.dim, self.dq), _pad_heads(t["uv"], H, spec.vdim, self.dv)
        self.w_ukv = put(torch.cat([uk, uv], 0))                       # keys of all heads, then values of all heads
        o = t["o"].view(-1, H, spec.vdim)
        if self.dv != spec.vdim:
            wide_o = torch.zeros(o.shape[0], H, self.dv, dtype=o.dtype, device=o.device)
            wide_o[:, :, :spec.vdim] = o
            o = wide_o
        self.w_o = put(o.reshape(o.shape[0], H * self.dv))

    @property
    def cache_rank(self) -> int:
        return self.spec.kv_rank

    def _expanded(self, q, seg, layer, cache, c, out):
        s, H = self.spec, self.spec.heads
        lo, n = seg.start, seg.sequences * seg.count
        if seg.begin == 0:
            ctx, length = c[lo:lo + n], seg.count
        else:
            length = seg.begin + seg.count
            ctx = cache.gather(layer, seg.slot, length)
        kv = linear(ctx, self.w_ukv).view(seg.sequences, length, 2, H, self.dq)
        shape = (seg.sequences, seg.count, H, self.dq)
        flash_forward(q[lo:lo + n].view(shape), kv[:, :, 0], kv[:, :, 1], causal=True, scale=s.scale, out=out[lo:lo + n].view(shape))

    def _latent(self, q, lo, batch, layer, cache, out):
        s, H, R = self.spec, self.spec.heads, self.spec.kv_rank
        n = q.shape[0] - lo
        wk = self.w_ukv[:H * self.dq].view(H, self.dq, R)
        wv = self.w_ukv[H * self.dq:].view(H, self.dv, R)
        qh = q[lo:].view(n, H, self.dq).transpose(0, 1)
        qa = torch.empty(n, H, R, dtype=q.dtype, device=q.device)
        linear(qh, wk, w_mn=True, out=qa.transpose(0, 1))
        ol = cache.attention(layer, qa, batch.slot[lo:], batch.pos[lo:], s.scale, batch.max_len)
        linear(ol.transpose(0, 1), wv, out=out[lo:].view(n, H, self.dv).transpose(0, 1))

    def forward(self, h: torch.Tensor, batch, cache, layer: int) -> torch.Tensor:
        """h [N, width], the tokens of ``batch``; appends their latents to layer ``layer`` of ``cache``."""
        s = self.spec
        lat = linear(h, self.w_down, out_dtype=torch.float32)
        segs = batch.prompts if self.prompt_form else ()
        split = batch.single_from if self.prompt_form else 0
        cq, c = cache.norm_append(layer, lat, self.q_norm, self.kv_norm, self.eps, batch.slot, batch.pos,
                                  keep=any(seg.begin == 0 for seg in segs))
        q = linear(cq, self.w_uq)
        o = torch.empty(h.shape[0], s.heads * self.dv, dtype=h.dtype, device=h.device)
        for seg in segs:
            self._expanded(q, seg, layer, cache, c, o)
        if split < h.shape[0]:
            self._latent(q, split, batch, layer, cache, o)
        return linear(o, self.w_o)
