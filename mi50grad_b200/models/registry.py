"""Model registry: which configuration reader, checkpoint loader and engine serve a
model directory, chosen by its config.json.

A config.json that names an `architecture` is looked up by that name; every other
one is a HuggingFace config of the Qwen3.5 hybrid decoder."""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable, Dict

DEFAULT = "Qwen3.5"


@dataclass(frozen=True)
class Architecture:
    name: str
    load_config: Callable        # (model_dir) -> config
    make_loader: Callable        # (model_dir, config or None) -> checkpoint loader
    make_engine: Callable        # (config, device_id, max_seq_len, **engine keywords) -> engine without weights
    dtypes: tuple                # element types an engine of this architecture can compute in
    tensor_parallel: bool


def _qwen_config(model_dir):
    from ..config import load_config_from_json
    return load_config_from_json(model_dir)


def _qwen_loader(model_dir, config=None):
    from ..loaders.checkpoint import CheckpointLoader
    return CheckpointLoader(model_dir, config)


def _qwen_engine(config, device_id=0, max_seq_len=2048, **kw):
    from ..engine.engine import InferenceEngine
    kw.pop("dtype", None)
    return InferenceEngine(config, device_id, max_seq_len, **kw)


def _degedra_config(model_dir):
    from ..loaders.mixer import load_degedra_config
    return load_degedra_config(model_dir)


def _degedra_loader(model_dir, config=None):
    from ..loaders.mixer import DegedraLoader
    return DegedraLoader(model_dir, config)


def _degedra_engine(config, device_id=0, max_seq_len=2048, **kw):
    from ..engine.mixer_engine import MixerEngine
    return MixerEngine(config, device_id, max_seq_len, **kw)


def _vekerax_config(model_dir):
    from ..loaders.mixer import load_vekerax_config
    return load_vekerax_config(model_dir)


def _vekerax_loader(model_dir, config=None):
    from ..loaders.mixer import VekeraxLoader
    return VekeraxLoader(model_dir, config)


def _vekerax_engine(config, device_id=0, max_seq_len=2048, **kw):
    from ..engine.vekerax_engine import VekeraxEngine
    return VekeraxEngine(config, device_id, max_seq_len, **kw)


ARCHITECTURES: Dict[str, Architecture] = {
    DEFAULT: Architecture(DEFAULT, _qwen_config, _qwen_loader, _qwen_engine, ("float16",), True),
    "Degedra": Architecture("Degedra", _degedra_config, _degedra_loader, _degedra_engine, ("bfloat16", "float32"), False),
    "Vekerax": Architecture("Vekerax", _vekerax_config, _vekerax_loader, _vekerax_engine, ("bfloat16", "float32"), False),
}


def architecture_of(model_dir: str) -> Architecture:
    path = Path(model_dir) / "config.json"
    if not path.exists():
        raise FileNotFoundError(f"No config.json found in {model_dir}")
    name = json.loads(path.read_text()).get("architecture", DEFAULT)
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[name]


def load_model_config(model_dir: str):
    return architecture_of(model_dir).load_config(model_dir)


def build_engine(model_dir: str, device_id: int = 0, max_seq_len: int = 2048, **kw):
    """Engine of one GPU with the directory's weights loaded -> (engine, loader)."""
    arch = architecture_of(model_dir)
    loader = arch.make_loader(model_dir)
    eng = arch.make_engine(loader.config, device_id, max_seq_len, **kw)
    for i in range(loader.config.num_hidden_layers):
        eng.load_layer_weights(i, loader.load_layer(i))
    eng.load_lm_head(loader.load_lm_head())
    eng.load_embedding(loader.load_embedding())
    eng.load_final_norm(loader.load_final_norm())
    return eng, loader
