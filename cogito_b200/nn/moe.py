"""Gated feed-forward layers of inference models: dense (act(gate) * up, act silu or relu) and mixture of experts with a softmax
router, an additive correction that steers the choice only, group-limited selection, identity outputs and a shared
expert that every token takes."""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..ops import moe as X
from ..ops.linear import gated_linear, linear
from .latent_attention import _frozen


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class MoESpec:
    expert_ff: int
    experts: int           # with weights
    top: int
    identity: int = 0      # router outputs after the experts that stand for the input itself
    groups: int = 1
    keep: int = 1          # groups whose outputs can be chosen
    shared_ff: int = 0     # 0: no shared expert

    @property
    def outputs(self) -> int:
        return self.experts + self.identity


class GatedMLP(nn.Module):
    """W_down (act(W_gate h) * (W_up h)); the gate and up products are one product."""

    def __init__(self, tensors, device, dtype, act: str = "silu"):
        super().__init__()
        t = {k: v.to(device) for k, v in tensors.items()}
        self.act = act
        self.w_gate_up = _frozen(torch.cat([t["gate"], t["up"]], 0).to(dtype).contiguous())
        self.w_down = _frozen(t["down"].to(dtype).contiguous())

    def inner(self, h, out=None):
        """act(W_gate h) * (W_up h), what W_down is applied to."""
        return gated_linear(h, self.w_gate_up, self.act, out)

    def forward(self, h):
        return linear(self.inner(h), self.w_down)

    def branch(self, h):
        """What the stream update adds: (dense result, no expert rows)."""
        return self.forward(h), {}


class MixtureOfExperts(nn.Module):
    def __init__(self, spec: MoESpec, tensors, device, dtype):
        super().__init__()
        self.spec = spec
        E = range(spec.experts)
        self.w_gate_up = _frozen(torch.stack([torch.cat([tensors[f"e{i}.gate"], tensors[f"e{i}.up"]], 0) for i in E]).to(device, dtype).contiguous())
        self.w_down = _frozen(torch.stack([tensors[f"e{i}.down"] for i in E]).to(device, dtype).contiguous())
        self.w_router = _frozen(tensors["router"].to(device, dtype).contiguous())
        self.correction = _frozen(tensors["correction"].to(device).float().contiguous())
        self.shared = None
        if spec.shared_ff:
            self.shared = GatedMLP({k: tensors[f"shared.{k}"] for k in ("gate", "up", "down")}, device, dtype)

    def branch(self, h):
        """(shared expert's result or None, the weighted expert rows as keyword arguments of ``stream_update``)."""
        s = self.spec
        logits = linear(h, self.w_router, out_dtype=torch.float32)
        grouped = X.grouped_ok(h, self.w_gate_up, self.w_down) and h.shape[0] * s.top > X.FEW_PAIRS
        r = X.route(logits, self.correction, s.experts, s.top, s.groups, s.keep, count=grouped)
        rows = X.expert_outputs(h, r, self.w_gate_up, self.w_down)
        y = self.shared(h) if self.shared is not None else None
        return y, {"pairs": rows, "row_of": r.row_of, "weight": r.weight}
