"""Angles of rotary positions (interleaved pairs), formed once per step and shared by every layer with the same rotation.
CUDA: csrc/kernels/kv_rows.cu; CPU tensors take the same steps in PyTorch."""
from __future__ import annotations

import math

import torch

from . import _lib


def frequencies(base: float, dims: int, device=None) -> torch.Tensor:
    """fp64 [dims / 2]: pair i turns by base^(-2i / dims) per position."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / max(dims, 1)).to(device)


def angles(pos: torch.Tensor, freq: torch.Tensor) -> torch.Tensor:
    """pos int32 [N], freq fp64 [n] -> fp32 [N, n, 2], (cos, sin) of pos * freq; the product is formed and reduced in fp64."""
    if not pos.is_cuda:
        a = pos.double()[:, None] * freq[None]
        a = (a - 2 * math.pi * torch.round(a / (2 * math.pi))).float()
        return torch.stack([torch.cos(a), torch.sin(a)], -1)
    out = torch.empty(pos.shape[0], freq.shape[0], 2, dtype=torch.float32, device=pos.device)
    _lib.check(_lib.lib().cgk_rotary_angles(pos.data_ptr(), freq.data_ptr(), out.data_ptr(), pos.shape[0], freq.shape[0], _lib.stream_ptr()),
               "cgk_rotary_angles")
    _lib.count_launch()
    return out


def turn(x: torch.Tensor, cs: torch.Tensor) -> torch.Tensor:
    """x fp32 [N, heads, D], cs [N, n, 2]: the first 2n elements of every head, pair by pair."""
    n = cs.shape[1]
    u, v, c, s = x[..., 0:2 * n:2], x[..., 1:2 * n:2], cs[:, None, :, 0], cs[:, None, :, 1]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., 2 * n:]], -1)
