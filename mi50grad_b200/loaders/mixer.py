"""Checkpoint reader of the Degedra decoder: config.json plus bf16 safetensors under
the names `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.*`, `l<i>.norm1/2`,
`embed`, `final.norm`, `head`."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, Optional

import torch

from ..config import DegedraConfig, degedra_config_from_dict
from ..models.mixer_weights import TENSOR_NAMES, MixerLayerWeights, MixerModelWeights, layer_shapes
from .safetensors_io import CheckpointDir


def load_degedra_config(model_dir: str) -> DegedraConfig:
    return degedra_config_from_dict(json.loads((Path(model_dir) / "config.json").read_text()))


class DegedraLoader:
    def __init__(self, model_dir: str, config: Optional[DegedraConfig] = None):
        self.model_dir = str(model_dir)
        self.config = config or load_degedra_config(model_dir)
        self.fmt = "bf16"
        self.ck = CheckpointDir(model_dir, lazy=True)
        self._layers: Dict[int, MixerLayerWeights] = {}

    def load_tensor(self, key: str, shape=None) -> torch.Tensor:
        t = self.ck.get(key, bf16_to=None)
        if shape is not None and tuple(t.shape) != tuple(shape):
            raise ValueError(f"{key}: shape {tuple(t.shape)}, expected {tuple(shape)}")
        return t

    def load_layer(self, layer_idx: int) -> MixerLayerWeights:
        j = self.config.weight_layer(layer_idx)
        if j not in self._layers:
            shapes = layer_shapes(self.config.hidden_size, self.config.layers[j])
            self._layers[j] = MixerLayerWeights(**{n: self.load_tensor(f"l{j}.{TENSOR_NAMES[n]}", sh)
                                                   for n, sh in shapes.items()})
        return self._layers[j]

    def load_embedding(self) -> torch.Tensor:
        return self.load_tensor("embed", (self.config.vocab_size, self.config.hidden_size))

    def load_lm_head(self) -> torch.Tensor:
        return self.load_tensor("head", (self.config.vocab_size, self.config.hidden_size))

    def load_final_norm(self) -> torch.Tensor:
        return self.load_tensor("final.norm", (self.config.hidden_size,))

    def load_model(self) -> MixerModelWeights:
        mw = MixerModelWeights(self.config)
        mw.layers = [self.load_layer(i) for i in range(self.config.num_hidden_layers)]
        mw.embed, mw.head, mw.final_norm = self.load_embedding(), self.load_lm_head(), self.load_final_norm()
        return mw

    def get_all_tensor_keys(self):
        return self.ck.keys()
