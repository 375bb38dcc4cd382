"""Surelorn: a decoder-only language model with latent attention (no rotary part; a sinusoidal position vector is
added to the scaled embedding), dense or mixture-of-experts feed-forward layers, RMS norms on the output of each
sublayer, and layers that may reuse another layer's weights with a cache of their own.

    x = scale * E[tok] + pos;   x += n1(attention(x));   x += n2(feed_forward(x));   logits = head n_final(x)

The stream x is fp32; matrix products take its bf16 copy (or fp32 throughout with ``dtype=torch.float32``).
Built from the mechanisms in ``nn.latent_attention``, ``nn.moe`` and ``ops.stream``; run by
``serve.stack.StackEngine``, which owns cache, batches and logits.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import torch
from torch import nn

from ..nn.latent_attention import LatentAttention, LatentSpec, _frozen
from ..nn.moe import DenseSpec, GatedMLP, MixtureOfExperts, MoESpec
from ..ops import stream as S
from ..ops.linear import linear
from ..serve.kv_cache import PagedLatentCache
from .registry import save_folder  # noqa: F401

POSITION_BASE = 10000.0


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentSpec
    mlp: DenseSpec | MoESpec | None
    weights_of: int | None = None


@dataclass(frozen=True)
class SurelornConfig:
    vocab_size: int
    width: int
    layers: tuple[LayerSpec, ...] = field(default_factory=tuple)
    embedding_scale: float = 1.0
    norm_eps: float = 1e-6

    architecture = "Surelorn"

    @classmethod
    def from_dict(cls, d: dict) -> "SurelornConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            m, mlp = e["mixer"], e.get("mlp")
            mixer = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]), float(m["scale"]))
            layers.append(LayerSpec(mixer, cls._mlp(i, mlp), e.get("weights_of")))
        cfg = cls(int(d["vocab"]), int(d["width"]), tuple(layers), float(d["embedding"]["scale"]), float(d["norm"]["eps"]))
        for i, l in enumerate(layers):
            h = layers[cfg.home(i)]
            if (l.mixer, l.mlp) != (h.mixer, h.mlp):
                raise ValueError(f"layer {i} uses the weights of layer {cfg.home(i)}, whose sizes differ")
        return cfg

    @staticmethod
    def _mlp(i, mlp):
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return DenseSpec(int(mlp["ff"]))
        if mlp["kind"] != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        r, groups, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
        s = MoESpec(int(mlp["expert"]["ff"]), int(r["experts"]), int(r["top"]), int(r.get("identity") or 0),
                    int(groups["count"]) if groups else 1, int(groups["keep"]) if groups else 1, int(shared["ff"]) if shared else 0)
        if s.outputs % s.groups or not 0 < s.keep <= s.groups or s.top > s.keep * (s.outputs // s.groups):
            raise ValueError(f"layer {i}: {s.outputs} router outputs in {s.groups} groups, {s.keep} kept, cannot give {s.top} choices")
        return s

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            e = {"type": "latent_attention", "mixer": {k: getattr(l.mixer, k) for k in ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale")}}
            if l.mlp is None:
                e["mlp"] = None
            elif isinstance(l.mlp, DenseSpec):
                e["mlp"] = {"kind": "dense", "ff": l.mlp.ff}
            else:
                router = {"experts": l.mlp.experts, "top": l.mlp.top, "identity": l.mlp.identity}
                if l.mlp.groups > 1:
                    router["groups"] = {"count": l.mlp.groups, "keep": l.mlp.keep}
                e["mlp"] = {"kind": "moe", "expert": {"ff": l.mlp.expert_ff}, "router": router}
                if l.mlp.shared_ff:
                    e["mlp"]["shared"] = {"ff": l.mlp.shared_ff}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            out.append(e)
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps}, "layers": out}

    def home(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            seen.add(i)
            j = self.layers[i].weights_of
            if not 0 <= j < len(self.layers) or j in seen:
                raise ValueError(f"layer {i}: weights_of {j} does not lead to a layer with tensors")
            i = j
        return i

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Names and shapes of a checkpoint, linear weights [out, in]."""
        W, out = self.width, {"embed": (self.vocab_size, self.width)}

        def gated(p, ff):
            out[p + "gate"], out[p + "up"], out[p + "down"] = (ff, W), (ff, W), (W, ff)
        for i, l in enumerate(self.layers):
            if l.weights_of is not None:
                continue
            p, m = f"l{i}.", l.mixer
            out[p + "norm1"] = (W,)
            out.update({p + "mix.dq": (m.q_rank, W), p + "mix.dq.norm": (m.q_rank,), p + "mix.uq": (m.heads * m.dim, m.q_rank),
                        p + "mix.dkv": (m.kv_rank, W), p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (m.heads * m.dim, m.kv_rank),
                        p + "mix.uv": (m.heads * m.vdim, m.kv_rank), p + "mix.o": (W, m.heads * m.vdim)})
            if l.mlp is None:
                continue
            out[p + "norm2"] = (W,)
            if isinstance(l.mlp, DenseSpec):
                gated(p + "mlp.", l.mlp.ff)
            else:
                for e in range(l.mlp.experts):
                    gated(f"{p}mlp.e{e}.", l.mlp.expert_ff)
                out[p + "mlp.router"], out[p + "mlp.correction"] = (l.mlp.outputs, W), (l.mlp.outputs,)
                if l.mlp.shared_ff:
                    gated(p + "mlp.shared.", l.mlp.shared_ff)
        out["final.norm"], out["head"] = (W,), (self.vocab_size, W)
        return out


def random_tensors(cfg: SurelornConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """bf16 checkpoint tensors: matrices N(0, 1 / in), norms around 1, small router corrections."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        t = torch.randn(shape, generator=g, device=device)
        if name.endswith("correction"):
            t = t * 0.02
        elif len(shape) == 1:
            t = 1.0 + 0.1 * t
        elif name != "embed":
            t = t * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


class _Layer(nn.Module):
    """One set of layer tensors."""

    def __init__(self, cfg: SurelornConfig, i: int, tensors, device, dtype):
        super().__init__()
        spec, p = cfg.layers[i], f"l{i}."

        def part(prefix):
            return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}
        norm = lambda name: _frozen(tensors[p + name].to(device).float().contiguous())
        self.attn = LatentAttention(spec.mixer, part(p + "mix."), cfg.norm_eps, device, dtype)
        self.norm1 = norm("norm1")
        self.mlp = None
        if spec.mlp is not None:
            t = part(p + "mlp.")
            self.mlp = GatedMLP(t, device, dtype) if isinstance(spec.mlp, DenseSpec) else MixtureOfExperts(spec.mlp, t, device, dtype)
            self.norm2 = norm("norm2")


class Surelorn(nn.Module):
    def __init__(self, cfg: SurelornConfig, tensors: dict[str, torch.Tensor] | None = None, device="cpu", dtype=torch.bfloat16):
        """tensors: a checkpoint as ``cfg.tensor_shapes`` names it (None: random weights)."""
        super().__init__()
        if tensors is None:
            tensors = random_tensors(cfg, device=device)
        want = cfg.tensor_shapes()
        bad = [k for k, s in want.items() if k not in tensors or tuple(tensors[k].shape) != tuple(s)]
        if bad:
            raise ValueError(f"checkpoint tensors missing or of another shape: {bad[:5]}")
        self.cfg, self.dtype = cfg, dtype
        self.device = torch.device(device)
        self.embed = _frozen(tensors["embed"].to(device, dtype).contiguous())
        self.head = _frozen(tensors["head"].to(device, dtype).contiguous())
        self.norm_f = _frozen(tensors["final.norm"].to(device).float().contiguous())
        self.sets = nn.ModuleDict({str(i): _Layer(cfg, i, tensors, device, dtype) for i, l in enumerate(cfg.layers) if l.weights_of is None})
        self.register_buffer("freq", S.sinusoid_frequencies(cfg.width, POSITION_BASE, device), persistent=False)
        self.runs = [self.sets[str(cfg.home(i))] for i in range(len(cfg.layers))]

    # ------------------------------------------------------------ what an engine asks of a model
    def new_cache(self, batch: int, max_seq_len: int, page_size: int, n_pages: int | None = None) -> PagedLatentCache:
        return PagedLatentCache([l.attn.cache_rank for l in self.runs], batch, max_seq_len, page_size, self.device, self.dtype, n_pages)

    def vocab(self) -> int:
        return self.cfg.vocab_size

    def stream(self, batch, cache, keep=None) -> torch.Tensor:
        """The residual stream [N, width] (fp32) of the tokens of ``batch`` after the last layer; their latents are
        appended to ``cache``.  keep: a list that receives a copy after every layer."""
        eps, dt = self.cfg.norm_eps, self.dtype
        x, h = S.embed_sinusoid(batch.ids, batch.pos, self.embed, self.cfg.embedding_scale, self.freq)
        for i, l in enumerate(self.runs):
            h = S.stream_update(x, l.attn(h, batch, cache, i), l.norm1, eps, dt)
            if l.mlp is not None:
                y, pairs = l.mlp.branch(h)
                h = S.stream_update(x, y, l.norm2, eps, dt, **pairs)
            if keep is not None:
                keep.append(x.clone())
        return x

    def logits(self, x: torch.Tensor, rows: torch.Tensor | None = None) -> torch.Tensor:
        """fp32 logits of the stream's rows (all, or those named)."""
        return linear(S.rms_rows(x, self.norm_f, self.cfg.norm_eps, self.dtype, rows), self.head, out_dtype=torch.float32)

    def num_params(self) -> int:
        return sum(p.numel() for p in self.parameters())

    # ------------------------------------------------------------ folders
    @classmethod
    def from_folder(cls, path: str, device="cpu", dtype=torch.bfloat16) -> "Surelorn":
        from ..io.safetensors import load_safetensors
        with open(os.path.join(path, "config.json")) as f:
            cfg = SurelornConfig.from_dict(json.load(f))
        return cls(cfg, load_safetensors(os.path.join(path, "model.safetensors")), device, dtype)

