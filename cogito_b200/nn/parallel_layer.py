"""A layer whose mixer and feed-forward read one residual stream through norms of their own:

    x <- x + m (mixer(n1(x)) + ff(n2(x)))

Their output products are one: the mixer's heads and the feed-forward's inner activations stand side by side in a row, and
so do the two matrices."""
from __future__ import annotations

import torch
from torch import nn

from ..ops.linear import linear
from .latent_attention import _frozen


def _ceil8(n: int) -> int:
    return (n + 7) // 8 * 8


def rows_of_8(w: torch.Tensor) -> torch.Tensor:
    """[n, K] with zero rows up to a multiple of 8."""
    return torch.nn.functional.pad(w, (0, 0, 0, _ceil8(w.shape[0]) - w.shape[0]))


class ParallelLayer(nn.Module):
    """mixer: a module with ``out_width`` that is called as mixer(h, batch, cache, layer, out); mlp: a ``GatedMLP`` or None;
    w_o: the mixer's output matrix [width, out_width]; norm1, norm2: fp32 norm weights (norm2 None without mlp)."""

    def __init__(self, mixer, mlp, w_o, norm1, norm2, device, dtype):
        super().__init__()
        self.mixer, self.mlp = mixer, mlp
        self.norm1 = _frozen(norm1.to(device).float().contiguous())
        self.norm2 = None if norm2 is None else _frozen(norm2.to(device).float().contiguous())
        # each part starts on 16 bytes: the row kernels and TMA want that; columns between the parts are zero in both factors
        n = w_o.shape[1]
        self.ff_at = _ceil8(n)
        self.ff = 0 if mlp is None else mlp.w_down.shape[1]
        w = torch.zeros(w_o.shape[0], self.ff_at + _ceil8(self.ff), dtype=dtype, device=device)
        w[:, :n] = w_o.to(device, dtype)
        if mlp is not None:
            w[:, self.ff_at:self.ff_at + self.ff] = mlp.w_down
            del mlp.w_down
        self.w_out = _frozen(w)
        self.gaps = w.shape[1] != n + self.ff

    def forward(self, h1, h2, batch, cache, layer: int) -> torch.Tensor:
        """The normed stream for the mixer and for the feed-forward -> mixer + feed-forward [N, width]."""
        rows = (torch.zeros if self.gaps else torch.empty)(h1.shape[0], self.w_out.shape[1], dtype=h1.dtype, device=h1.device)
        self.mixer(h1, batch, cache, layer, rows[:, :self.mixer.out_width])
        if self.mlp is not None:
            self.mlp.inner(h2, rows[:, self.ff_at:self.ff_at + self.ff])
        return linear(rows, self.w_out, out_dtype=h1.dtype)
