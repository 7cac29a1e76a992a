"""Weights of the post-norm decoders of parallel mixers: the per-layer bundle the
engine consumes, random initialisation, and the checkpoint writer.

Tensors keep the checkpoint's layout ([out, in] matrices, bf16); the engine packs
them (fused in-projection, common output projection, gate / up interleaved).
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field, fields
from pathlib import Path
from typing import Dict, List, Optional, Tuple

import torch

from ..config import DegedraConfig, ParallelLayerSpec, degedra_config_to_dict

# field of MixerLayerWeights -> tensor name behind "l<i>."
TENSOR_NAMES = {
    "norm1": "norm1", "norm2": "norm2",
    "q": "mix.left.q", "k": "mix.left.k", "q_norm": "mix.left.q.norm", "k_norm": "mix.left.k.norm", "attn_o": "mix.left.o",
    "ssd_in": "mix.right.in", "conv": "mix.right.conv", "conv_b": "mix.right.conv.b", "dt_bias": "mix.right.dt_bias",
    "A_log": "mix.right.A_log", "D": "mix.right.D", "ssd_norm": "mix.right.norm", "ssd_o": "mix.right.o",
    "gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down",
}


@dataclass
class MixerLayerWeights:
    norm1: torch.Tensor
    q: torch.Tensor
    k: torch.Tensor
    q_norm: torch.Tensor
    k_norm: torch.Tensor
    attn_o: torch.Tensor
    ssd_in: torch.Tensor
    conv: torch.Tensor
    conv_b: torch.Tensor
    dt_bias: torch.Tensor
    A_log: torch.Tensor
    D: torch.Tensor
    ssd_norm: torch.Tensor
    ssd_o: torch.Tensor
    norm2: Optional[torch.Tensor] = None
    gate: Optional[torch.Tensor] = None
    up: Optional[torch.Tensor] = None
    down: Optional[torch.Tensor] = None


@dataclass
class MixerModelWeights:
    """`layers[i]` of a layer that uses another layer's tensors is that layer's object."""
    config: DegedraConfig
    layers: List[MixerLayerWeights] = field(default_factory=list)
    embed: Optional[torch.Tensor] = None
    head: Optional[torch.Tensor] = None
    final_norm: Optional[torch.Tensor] = None


def layer_shapes(width: int, l: ParallelLayerSpec) -> Dict[str, Tuple[int, ...]]:
    a, s = l.attention, l.ssd
    sh = {
        "norm1": (width,), "q": (a.heads * a.dim, width), "k": (a.kv_heads * a.dim, width),
        "q_norm": (a.heads * a.dim,), "k_norm": (a.kv_heads * a.dim,), "attn_o": (width, a.heads * a.dim),
        "ssd_in": (s.inner + s.conv_channels + s.heads, width), "conv": (s.conv_channels, s.conv), "conv_b": (s.conv_channels,),
        "dt_bias": (s.heads,), "A_log": (s.heads,), "D": (s.heads,), "ssd_norm": (s.inner,), "ssd_o": (width, s.inner),
    }
    if l.ff:
        sh.update(norm2=(width,), gate=(l.ff, width), up=(l.ff, width), down=(width, l.ff))
    return sh


def random_mixer_model(cfg: DegedraConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> MixerModelWeights:
    """Matrices of standard deviation 1/sqrt(fan-in), norm weights around one, step sizes and decay rates
    spread over the range a trained recurrence uses."""
    gen = torch.Generator(device=device)
    gen.manual_seed(seed)
    rnd = lambda *sh, std=1.0: torch.randn(*sh, generator=gen, device=device) * std
    mw = MixerModelWeights(cfg)
    for i, l in enumerate(cfg.layers):
        j = cfg.weight_layer(i)
        if j != i:
            mw.layers.append(None)
            continue
        t = {}
        for n, sh in layer_shapes(cfg.hidden_size, l).items():
            if n.endswith("norm") or n in ("norm1", "norm2"):
                v = 1.0 + rnd(*sh, std=0.1)
            elif n == "dt_bias":
                v = rnd(*sh, std=0.7) - 2.0
            elif n == "A_log":
                v = torch.rand(*sh, generator=gen, device=device) * 2.5
            elif n == "D":
                v = 1.0 + rnd(*sh, std=0.3)
            elif n == "conv":
                v = rnd(*sh, std=sh[1] ** -0.5)
            elif n == "conv_b":
                v = rnd(*sh, std=0.2)
            else:
                v = rnd(*sh, std=sh[1] ** -0.5)
            t[n] = v.to(dtype)
        mw.layers.append(MixerLayerWeights(**t))
    for i in range(len(mw.layers)):
        mw.layers[i] = mw.layers[cfg.weight_layer(i)]
    mw.embed = rnd(cfg.vocab_size, cfg.hidden_size).to(dtype)
    mw.head = rnd(cfg.vocab_size, cfg.hidden_size, std=2.0 * cfg.hidden_size ** -0.5).to(dtype)
    mw.final_norm = (1.0 + rnd(cfg.hidden_size, std=0.1)).to(dtype)
    return mw


def named_tensors(mw: MixerModelWeights) -> Dict[str, torch.Tensor]:
    out = {"embed": mw.embed, "head": mw.head, "final.norm": mw.final_norm}
    for i, lw in enumerate(mw.layers):
        if mw.config.weight_layer(i) != i:
            continue
        for f in fields(lw):
            v = getattr(lw, f.name)
            if v is not None:
                out[f"l{i}.{TENSOR_NAMES[f.name]}"] = v
    return out


def write_mixer_checkpoint(mw: MixerModelWeights, out_dir: str) -> None:
    from ..loaders.safetensors_io import save_safetensors
    out = Path(out_dir)
    out.mkdir(parents=True, exist_ok=True)
    (out / "config.json").write_text(json.dumps(degedra_config_to_dict(mw.config), indent=1))
    save_safetensors(str(out / "model.safetensors"), named_tensors(mw))
