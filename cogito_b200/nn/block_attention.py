"""Grouped-query attention with rotary positions over a paged cache, for the layer-stack engine.  What a design may choose
is in ``AttentionSpec``: positions that only see their own block, a sink in the softmax denominator, values that are
RMS-normed, values that are turned by their position (and the result turned back by the query's), keys and values of
another layer.

Two forms.  Prompt portions use the flash-attention kernel on contiguous keys and values (gathered from the pages where a
portion continues a block).  Single tokens, short portions, heads longer than 128 and fp32 read the pages directly.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..ops import rotary
from ..ops.attention import flash_forward
from ..ops.linear import linear
from .latent_attention import _frozen
from .parallel_layer import rows_of_8


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                      # query / key elements per head
    vdim: int                     # value elements per head
    scale: float                  # of the scores
    rot_base: float = 10000.0
    rot_dims: int = 0             # elements of a query / key head that are turned (interleaved pairs)
    block: int = 0                # positions that see each other; 0: all earlier ones
    sink: bool = False
    norm_values: bool = False
    turn_values: bool = False
    kv_from: int | None = None    # the layer whose keys and values are used


def step_angles(batch, freq):
    """(cos, sin) of the step's tokens, formed once per step and rotation."""
    key = ("angles", freq.data_ptr())
    if key not in batch.memo:
        batch.memo[key] = rotary.angles(batch.pos, freq)
    return batch.memo[key]


class BlockAttention(nn.Module):
    """Inference module.  ``tensors``: q, k, v as [out, in] matrices (k and v absent with kv_from).  ``rotations``: shared
    frequency tables by (base, dims), so that layers with one rotation share a step's angles."""

    def __init__(self, spec: AttentionSpec, tensors: dict[str, torch.Tensor], eps: float, device, dtype, rotations: dict):
        super().__init__()
        self.spec, self.eps = spec, eps
        self.own = spec.kv_from is None
        parts = [tensors["q"]] + ([tensors["k"], tensors["v"]] if self.own else [])
        self.w_in = _frozen(rows_of_8(torch.cat([p.to(device) for p in parts], 0)).to(dtype).contiguous())
        wide = max(spec.dim, spec.vdim)
        # the flash kernel takes heads of 64 or 128 elements: shorter ones get zero columns (exact)
        self.prompt_form = dtype == torch.bfloat16 and wide <= 128
        self.wide = (64 if wide <= 64 else 128) if self.prompt_form else (spec.dim + 7) // 8 * 8

        def table(dims):
            key = (spec.rot_base, dims)
            if key not in rotations:
                rotations[key] = rotary.frequencies(spec.rot_base, dims, device)
            return rotations[key]
        self.freq_k = table(spec.rot_dims) if spec.rot_dims else None
        self.freq_v = table(spec.vdim) if spec.turn_values else None

    @property
    def out_width(self) -> int:
        return self.spec.heads * self.spec.vdim

    def forward(self, h: torch.Tensor, batch, cache, layer: int, out: torch.Tensor) -> torch.Tensor:
        """h [N, width], the tokens of ``batch``; writes the heads' results (before the output product) to ``out``
        [N, heads * vdim] and the keys and values, if they are the layer's own, to ``cache``."""
        s, N = self.spec, h.shape[0]
        x = linear(h, self.w_in, out_dtype=h.dtype)
        nq, nk = s.heads * s.dim, s.kv_heads * s.dim
        cs_k = None if self.freq_k is None else step_angles(batch, self.freq_k)
        cs_v = None if self.freq_v is None else step_angles(batch, self.freq_v)
        segs = batch.prompts if self.prompt_form else ()
        split = batch.single_from if self.prompt_form else 0
        k, v = (x[:, nq:nq + nk], x[:, nq + nk:nq + nk + s.kv_heads * s.vdim]) if self.own else (None, None)
        first = {id(g): g.begin // s.block * s.block if s.block else 0 for g in segs}
        q, kc, vc = cache.rotate_append(layer, x[:, :nq], k, v, cs_k, cs_v, s.heads, self.wide, batch.slot, batch.pos,
                                        self.eps if s.norm_values else None, keep=any(first[id(g)] == g.begin for g in segs))
        if self.own:
            batch.memo["kv", layer] = kc, vc
        else:
            kc, vc = batch.memo.get(("kv", s.kv_from), (None, None))
        for g in segs:
            lo, n = g.start, g.sequences * g.count
            if first[id(g)] == g.begin and kc is not None:
                kv = [t[lo:lo + n].view(g.sequences, g.count, s.kv_heads, self.wide) for t in (kc, vc)]
            else:
                kv = [t[None] for t in cache.gather(layer, g.slot, first[id(g)], g.begin + g.count - first[id(g)], self.wide)]
            flash_forward(q[lo:lo + n].view(g.sequences, g.count, s.heads, self.wide), *kv, causal=True, scale=s.scale, block=s.block, sink=s.sink,
                          turn=None if cs_v is None else cs_v[lo:lo + n].view(g.sequences, g.count, -1, 2),
                          out=out[lo:lo + n].unflatten(0, (g.sequences, g.count)).unflatten(-1, (s.heads, s.vdim)))
        if split < N:
            cache.attention(layer, q[split:], batch.slot[split:], batch.pos[split:], s.scale, batch.max_len, out[split:], s.block, s.sink,
                            None if cs_v is None else cs_v[split:])
        return out
