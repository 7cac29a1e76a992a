"""Weights of the Vekerax decoder: the per-layer bundle the engine consumes, random
initialisation, and the checkpoint writer.  Tensors keep the checkpoint's layout
([out, in] matrices, bf16); the engine packs them."""
from __future__ import annotations

import json
from dataclasses import dataclass, field, fields
from pathlib import Path
from typing import Dict, List, Optional, Tuple

import torch

from ..config import StreamLayerSpec, VekeraxConfig, vekerax_config_to_dict

# field of VekeraxLayerWeights -> tensor name behind "l<i>."
TENSOR_NAMES = {
    "norm1": "norm1", "norm2": "norm2", "q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o",
    "q_norm": "mix.q.norm", "k_norm": "mix.k.norm", "sink": "mix.sink", "g": "mix.g", "out_norm": "mix.norm",
    "gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down",
    "hc1_in": "hc1.in", "hc1_out": "hc1.out", "hc1_mix": "hc1.mix", "hc2_in": "hc2.in", "hc2_out": "hc2.out", "hc2_mix": "hc2.mix",
}


@dataclass
class VekeraxLayerWeights:
    norm1: torch.Tensor
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    o: torch.Tensor
    q_norm: Optional[torch.Tensor] = None       # attention
    k_norm: Optional[torch.Tensor] = None
    sink: Optional[torch.Tensor] = None
    g: Optional[torch.Tensor] = None            # lightning attention
    out_norm: Optional[torch.Tensor] = None
    norm2: Optional[torch.Tensor] = None        # feed-forward
    gate: Optional[torch.Tensor] = None
    up: Optional[torch.Tensor] = None
    down: Optional[torch.Tensor] = None
    hc1_in: Optional[torch.Tensor] = None       # hyper-connections of the mixer and of the feed-forward
    hc1_out: Optional[torch.Tensor] = None
    hc1_mix: Optional[torch.Tensor] = None
    hc2_in: Optional[torch.Tensor] = None
    hc2_out: Optional[torch.Tensor] = None
    hc2_mix: Optional[torch.Tensor] = None


@dataclass
class VekeraxModelWeights:
    """The output head is the embedding table."""
    config: VekeraxConfig
    layers: List[VekeraxLayerWeights] = field(default_factory=list)
    embed: Optional[torch.Tensor] = None
    final_norm: Optional[torch.Tensor] = None

    @property
    def head(self) -> Optional[torch.Tensor]:
        return self.embed


def layer_shapes(cfg: VekeraxConfig, l: StreamLayerSpec) -> Dict[str, Tuple[int, ...]]:
    w, n = cfg.hidden_size, cfg.streams
    if l.attention is not None:
        a = l.attention
        sh = {"q": (a.heads * a.dim, w), "k": (a.kv_heads * a.dim, w), "v": (a.kv_heads * a.vd, w), "o": (w, a.heads * a.vd),
              "q_norm": (a.dim,), "k_norm": (a.dim,), "sink": (a.heads,)}
    else:
        r = l.recurrence
        sh = {"q": (r.heads * r.state, w), "k": (r.heads * r.state, w), "v": (r.inner, w), "g": (r.inner, w), "o": (w, r.inner),
              "out_norm": (r.inner,)}
    sh["norm1"] = (w,)
    if l.ff:
        sh.update(norm2=(w,), gate=(l.ff, w), up=(l.ff, w), down=(w, l.ff))
    for q in ((1, 2) if l.ff else (1,)) if n else ():
        sh.update({f"hc{q}_in": (n,), f"hc{q}_out": (n,), f"hc{q}_mix": (n, n)})
    return sh


def random_vekerax_model(cfg: VekeraxConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> VekeraxModelWeights:
    """Matrices of standard deviation 1/sqrt(fan-in), norm weights around one, streams that keep most of
    themselves."""
    gen = torch.Generator(device=device)
    gen.manual_seed(seed)
    rnd = lambda *sh, std=1.0: torch.randn(*sh, generator=gen, device=device) * std
    mw = VekeraxModelWeights(cfg)
    for l in cfg.layers:
        t = {}
        for n, sh in layer_shapes(cfg, l).items():
            if "norm" in n:
                v = 1.0 + rnd(*sh, std=0.1)
            elif n.endswith("_mix"):
                v = 0.8 * torch.eye(sh[0], device=device) + rnd(*sh, std=0.3 / sh[0])
            elif n.startswith("hc"):
                v = (1.0 / sh[0] if n.endswith("_in") else 1.0) * (1.0 + rnd(*sh, std=0.3))
            elif n == "sink":
                v = rnd(*sh)
            else:
                v = rnd(*sh, std=sh[1] ** -0.5)
            t[n] = v.to(dtype)
        mw.layers.append(VekeraxLayerWeights(**t))
    mw.embed = rnd(cfg.vocab_size, cfg.hidden_size, std=cfg.hidden_size ** -0.5).to(dtype)
    mw.final_norm = (1.0 + rnd(cfg.hidden_size, std=0.1)).to(dtype)
    return mw


def named_tensors(mw: VekeraxModelWeights) -> Dict[str, torch.Tensor]:
    out = {"embed": mw.embed, "final.norm": mw.final_norm}
    for i, lw in enumerate(mw.layers):
        for f in fields(lw):
            v = getattr(lw, f.name)
            if v is not None:
                out[f"l{i}.{TENSOR_NAMES[f.name]}"] = v
    return out


def write_vekerax_checkpoint(mw: VekeraxModelWeights, out_dir: str) -> None:
    from ..loaders.safetensors_io import save_safetensors
    out = Path(out_dir)
    out.mkdir(parents=True, exist_ok=True)
    (out / "config.json").write_text(json.dumps(vekerax_config_to_dict(mw.config), indent=1))
    save_safetensors(str(out / "model.safetensors"), named_tensors(mw))
