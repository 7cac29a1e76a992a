"""Checkpoint readers of the decoders whose layers are described one by one:
config.json plus bf16 safetensors.

Degedra: `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.*`, `l<i>.norm1/2`, `embed`,
`final.norm`, `head`.  Vekerax: `l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.norm1/2`,
`l<i>.hc1/2.*`, `embed` (also the output head), `final.norm`."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, Optional

import torch

from ..config import DegedraConfig, VekeraxConfig, degedra_config_from_dict, vekerax_config_from_dict
from ..models import mixer_weights, vekerax_weights
from .safetensors_io import CheckpointDir


def load_degedra_config(model_dir: str) -> DegedraConfig:
    return degedra_config_from_dict(json.loads((Path(model_dir) / "config.json").read_text()))


def load_vekerax_config(model_dir: str) -> VekeraxConfig:
    return vekerax_config_from_dict(json.loads((Path(model_dir) / "config.json").read_text()))


class MixerCheckpoint:
    """Tensors of a checkpoint, checked against the shapes the configuration implies."""
    head_tensor = "head"

    def __init__(self, model_dir: str, config=None):
        self.model_dir = str(model_dir)
        self.config = config or self.read_config(model_dir)
        self.fmt = "bf16"
        self.ck = CheckpointDir(model_dir, lazy=True)
        self._layers: Dict[int, object] = {}

    def load_tensor(self, key: str, shape=None) -> torch.Tensor:
        t = self.ck.get(key, bf16_to=None)
        if shape is not None and tuple(t.shape) != tuple(shape):
            raise ValueError(f"{key}: shape {tuple(t.shape)}, expected {tuple(shape)}")
        return t

    def _layer(self, j: int, weights_type, names: dict, shapes: dict):
        if j not in self._layers:
            self._layers[j] = weights_type(**{n: self.load_tensor(f"l{j}.{names[n]}", sh) for n, sh in shapes.items()})
        return self._layers[j]

    def load_embedding(self) -> torch.Tensor:
        return self.load_tensor("embed", (self.config.vocab_size, self.config.hidden_size))

    def load_lm_head(self) -> torch.Tensor:
        return self.load_tensor(self.head_tensor, (self.config.vocab_size, self.config.hidden_size))

    def load_final_norm(self) -> torch.Tensor:
        return self.load_tensor("final.norm", (self.config.hidden_size,))

    def get_all_tensor_keys(self):
        return self.ck.keys()


class DegedraLoader(MixerCheckpoint):
    read_config = staticmethod(load_degedra_config)

    def __init__(self, model_dir: str, config: Optional[DegedraConfig] = None):
        super().__init__(model_dir, config)

    def load_layer(self, layer_idx: int) -> mixer_weights.MixerLayerWeights:
        j = self.config.weight_layer(layer_idx)
        return self._layer(j, mixer_weights.MixerLayerWeights, mixer_weights.TENSOR_NAMES,
                           mixer_weights.layer_shapes(self.config.hidden_size, self.config.layers[j]))

    def load_model(self) -> mixer_weights.MixerModelWeights:
        mw = mixer_weights.MixerModelWeights(self.config)
        mw.layers = [self.load_layer(i) for i in range(self.config.num_hidden_layers)]
        mw.embed, mw.head, mw.final_norm = self.load_embedding(), self.load_lm_head(), self.load_final_norm()
        return mw


class VekeraxLoader(MixerCheckpoint):
    read_config = staticmethod(load_vekerax_config)
    head_tensor = "embed"

    def __init__(self, model_dir: str, config: Optional[VekeraxConfig] = None):
        super().__init__(model_dir, config)

    def load_layer(self, layer_idx: int) -> vekerax_weights.VekeraxLayerWeights:
        return self._layer(layer_idx, vekerax_weights.VekeraxLayerWeights, vekerax_weights.TENSOR_NAMES,
                           vekerax_weights.layer_shapes(self.config, self.config.layers[layer_idx]))

    def load_model(self) -> vekerax_weights.VekeraxModelWeights:
        mw = vekerax_weights.VekeraxModelWeights(self.config)
        mw.layers = [self.load_layer(i) for i in range(self.config.num_hidden_layers)]
        mw.embed, mw.final_norm = self.load_embedding(), self.load_final_norm()
        return mw
