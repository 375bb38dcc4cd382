"""Model families by name.

``train`` families are built from the ``model`` section of a run configuration; ``serve`` architectures are
loaded from a folder whose ``config.json`` names them (key ``architecture``).  Modules are imported on first use.
"""
from __future__ import annotations

import importlib
import json
import os


def _cls(path: str):
    module, name = path.rsplit(":", 1)
    return getattr(importlib.import_module(f"cogito_b200.{module}"), name)


def _gpt2(m):
    return _cls("models.gpt2:GPT2Config")(vocab_size=m["vocab_size"], n_layer=m["n_layer"], d_model=m["d_model"], n_head=m["n_head"],
                                          d_ff=m["d_ff"], max_seq_len=m["max_seq_len"])


def _llama(m):
    return _cls("models.llama:LlamaConfig")(vocab_size=m["vocab_size"], n_layer=m["n_layer"], d_model=m["d_model"], n_head=m["n_head"],
                                            n_kv_head=m["n_kv_head"] or m["n_head"], d_ff=m["d_ff"], max_seq_len=m["max_seq_len"])


# family -> (configuration from a ``model`` section or None, model from (configuration or section, device, dtype))
TRAIN = {
    "gpt2": (_gpt2, lambda c, dev, dt: _cls("models.gpt2:GPT2")(c, device=dev, dtype=dt)),
    "llama": (_llama, lambda c, dev, dt: _cls("models.llama:Llama")(c, device=dev, dtype=dt)),
    "mlp": (None, lambda m, dev, dt: _cls("models.mlp:MLPClassifier")(m["in_features"], m["hidden"], m["classes"], device=dev, dtype=dt)),
    "cnn": (None, lambda m, dev, dt: _cls("models.cnn:ConvClassifier")(m["in_channels"], m["image"], m["channels"], m["classes"],
                                                                       device=dev, dtype=dt)),
}
# architecture -> class with ``from_folder(path, device, dtype)``; these run in serve.stack.StackEngine
SERVE = {"Surelorn": "models.surelorn:Surelorn", "Nufalorn": "models.nufalorn:Nufalorn"}


def train_config(family: str, section: dict):
    """Configuration object of a family's model (the section itself for families without one)."""
    if family not in TRAIN:
        raise SystemExit(f"unknown model.family {family}")
    make = TRAIN[family][0]
    return make(section) if make else section


def train_model(family: str, section: dict, device, dtype):
    return TRAIN[family][1](train_config(family, section), device, dtype) if family in TRAIN else train_config(family, section)


def load_folder(path: str, device="cuda", dtype=None):
    """The model in ``path`` (config.json + model.safetensors), its class chosen by config.json."""
    with open(os.path.join(path, "config.json")) as f:
        name = json.load(f).get("architecture")
    if name not in SERVE:
        raise ValueError(f"{path}: no model class for architecture {name!r} (known: {', '.join(SERVE)})")
    kw = {} if dtype is None else {"dtype": dtype}
    return _cls(SERVE[name]).from_folder(path, device, **kw)


def save_folder(path: str, cfg, tensors) -> None:
    """Writes config.json (``cfg.to_dict()``) and model.safetensors, what ``load_folder`` reads."""
    from ..io.safetensors import save_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg.to_dict(), f, indent=1)
    save_safetensors(os.path.join(path, "model.safetensors"), tensors)
