"""Model and engine configuration.

`QwenConfig` carries every dimension of the Qwen3.5 hybrid decoder (Gated
DeltaNet + gated full attention) with the same field names and defaults as the
reference's dataclass (reference: src/model/qwen.py:26-115), plus the JSON
loader for HuggingFace `config.json` files (reference: src/model/qwen.py:140-192)
and the memory estimators (reference: src/model/qwen.py:195-253), re-sized for a
180 GB B200 instead of a 16/32 GB MI50.

`EngineConfig` replaces the reference's ~20 imperative `set_*` toggles
(reference: src/inference/tp_engine.py:2252-2527) with one frozen description
of how the engine runs; the `set_*` names survive as thin shims on the engines.
"""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass, field
from pathlib import Path
from typing import List, Optional

B200_HBM_BYTES = 180 * 10**9


@dataclass
class QwenConfig:
    hidden_size: int = 5120
    intermediate_size: int = 17408
    num_hidden_layers: int = 64
    num_attention_heads: int = 24
    num_key_value_heads: int = 4
    head_dim: int = 256
    vocab_size: int = 248320
    max_position_embeddings: int = 262144
    rope_theta: float = 10000000.0
    rms_norm_eps: float = 1e-6

    full_attention_interval: int = 4
    layer_types: List[str] = field(default_factory=list)

    linear_key_head_dim: int = 128
    linear_num_key_heads: int = 16
    linear_num_value_heads: int = 48
    linear_value_head_dim: int = 128
    linear_conv_kernel_dim: int = 4

    partial_rotary_factor: float = 0.25
    mrope_sections: List[int] = field(default_factory=lambda: [11, 11, 10])
    mrope_interleaved: bool = True
    # 'interleaved' rotates pairs (2i, 2i+1) as the reference kernels do
    # (reference: src/kernels/qknorm_rope.hip:140-152); 'half' rotates
    # (i, i + rot/2) like HuggingFace's rotate_half.
    rope_style: str = "interleaved"

    quant_method: str = "gptq"
    bits: int = 4
    group_size: int = 128
    quant_sym: bool = True
    attn_quantized: bool = False

    attn_output_gate: bool = True

    def __post_init__(self):
        if not self.layer_types:
            self.layer_types = [
                "full_attention" if (i + 1) % self.full_attention_interval == 0
                else "linear_attention"
                for i in range(self.num_hidden_layers)
            ]
        if len(self.layer_types) != self.num_hidden_layers:
            raise ValueError("layer_types length must equal num_hidden_layers")

    # -- layer kinds -----------------------------------------------------
    def is_full_attention(self, layer_idx: int) -> bool:
        return self.layer_types[layer_idx] == "full_attention"

    def is_linear_attention(self, layer_idx: int) -> bool:
        return self.layer_types[layer_idx] == "linear_attention"

    @property
    def num_full_attention_layers(self) -> int:
        return sum(t == "full_attention" for t in self.layer_types)

    @property
    def num_linear_attention_layers(self) -> int:
        return sum(t == "linear_attention" for t in self.layer_types)

    # -- derived dims ------------------------------------------------------
    @property
    def full_attn_q_dim(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def full_attn_kv_dim(self) -> int:
        return self.num_key_value_heads * self.head_dim

    @property
    def linear_attn_key_dim(self) -> int:
        return self.linear_num_key_heads * self.linear_key_head_dim

    @property
    def linear_attn_value_dim(self) -> int:
        return self.linear_num_value_heads * self.linear_value_head_dim

    @property
    def linear_conv_dim(self) -> int:
        return 2 * self.linear_attn_key_dim + self.linear_attn_value_dim

    @property
    def kv_heads_per_group(self) -> int:
        return self.num_attention_heads // self.num_key_value_heads

    @property
    def rotary_dim(self) -> int:
        return int(self.head_dim * self.partial_rotary_factor)

    def full_attention_layer_indices(self) -> List[int]:
        return [i for i, t in enumerate(self.layer_types) if t == "full_attention"]

    def linear_attention_layer_indices(self) -> List[int]:
        return [i for i, t in enumerate(self.layer_types) if t == "linear_attention"]

    def max_tp(self) -> int:
        """Largest tensor-parallel degree the head counts allow.  KV heads are
        replicated when tp > num_key_value_heads, so the bound comes from the
        query heads, the DeltaNet key heads and the FFN width."""
        tp = 1
        while True:
            nxt = tp * 2
            if (self.num_attention_heads % nxt or self.linear_num_key_heads % nxt
                    or self.linear_num_value_heads % nxt
                    or self.intermediate_size % (8 * nxt)):
                return tp
            tp = nxt


def qwen35_27b(**overrides) -> QwenConfig:
    """The Qwen3.5-27B architecture the headline benchmark names."""
    return QwenConfig(**overrides)


def tiny_config(**overrides) -> QwenConfig:
    """The 4-layer CPU plumbing model: 3 Gated DeltaNet + 1 gated full-attention
    layer, hidden 256, FFN 704, 4 Q / 2 KV heads of 64, DeltaNet 2 QK / 4 V
    heads of 64, vocab 1024, partial RoPE over 16 dims, theta 1e7."""
    kw = dict(
        hidden_size=256, intermediate_size=704, num_hidden_layers=4,
        num_attention_heads=4, num_key_value_heads=2, head_dim=64,
        vocab_size=1024, max_position_embeddings=4096, rope_theta=1e7,
        rms_norm_eps=1e-6, full_attention_interval=4,
        linear_key_head_dim=64, linear_num_key_heads=2,
        linear_num_value_heads=4, linear_value_head_dim=64,
        linear_conv_kernel_dim=4, partial_rotary_factor=0.25,
        group_size=128, attn_quantized=True,
    )
    kw.update(overrides)
    return QwenConfig(**kw)


# (M, N, K, name) GEMM/GEMV shapes of the 27B model, used by the tuner and the
# micro-benchmarks (reference: src/model/qwen.py:117-137).
QWEN_GEMM_SHAPES = [
    (1, 2 * 6144 + 2 * 1024, 5120, "full_attn_qkv"),
    (512, 2 * 6144 + 2 * 1024, 5120, "full_attn_qkv_512"),
    (1, 2 * 2048 + 2 * 6144, 5120, "linear_attn_in_proj"),
    (512, 2 * 2048 + 2 * 6144, 5120, "linear_attn_in_proj_512"),
    (1, 5120, 6144, "attn_out_proj"),
    (512, 5120, 6144, "attn_out_proj_512"),
    (1, 2 * 17408, 5120, "ffn_gate_up"),
    (512, 2 * 17408, 5120, "ffn_gate_up_512"),
    (1, 5120, 17408, "ffn_down"),
    (512, 5120, 17408, "ffn_down_512"),
    (1, 248320, 5120, "lm_head"),
]


def load_config_from_json(model_dir: str) -> QwenConfig:
    path = Path(model_dir) / "config.json"
    if not path.exists():
        raise FileNotFoundError(f"No config.json found in {model_dir}")
    hf = json.loads(path.read_text())
    text = hf.get("text_config", hf)
    rope = text.get("rope_parameters", {}) or {}
    names = {f.name for f in dataclasses.fields(QwenConfig)}
    kw = {k: text[k] for k in (
        "hidden_size", "intermediate_size", "num_hidden_layers",
        "num_attention_heads", "num_key_value_heads", "head_dim", "vocab_size",
        "max_position_embeddings", "rms_norm_eps", "full_attention_interval",
        "linear_key_head_dim", "linear_num_key_heads", "linear_num_value_heads",
        "linear_value_head_dim", "linear_conv_kernel_dim", "attn_output_gate",
        "rope_style",
    ) if k in text and k in names}
    if text.get("layer_types"):
        kw["layer_types"] = list(text["layer_types"])
    kw["rope_theta"] = rope.get("rope_theta", text.get("rope_theta", 1e7))
    kw["partial_rotary_factor"] = rope.get(
        "partial_rotary_factor", text.get("partial_rotary_factor", 0.25))
    if "mrope_section" in rope:
        kw["mrope_sections"] = list(rope["mrope_section"])
    kw["mrope_interleaved"] = rope.get("mrope_interleaved", True)
    cfg = QwenConfig(**kw)
    q = hf.get("quantization_config", text.get("quantization_config", {})) or {}
    if q:
        cfg.quant_method = q.get("quant_method", "gptq")
        cfg.bits = q.get("bits", q.get("num_bits", 4))
        cfg.group_size = q.get("group_size", 128)
        for grp in (q.get("config_groups") or {}).values():
            w = grp.get("weights", {}) or {}
            cfg.bits = w.get("num_bits", cfg.bits)
            cfg.group_size = w.get("group_size", cfg.group_size)
            cfg.quant_sym = w.get("symmetric", cfg.quant_sym)
        cfg.quant_sym = q.get("sym", True)
        dyn = q.get("dynamic", {}) or {}
        cfg.attn_quantized = "-:.*attn.*" not in dyn
    return cfg


def kv_cache_bytes(config: QwenConfig, max_seq_len: int, batch: int = 1,
                   tp_size: int = 1) -> int:
    """Bytes of fp16 K+V cache per rank.  Only full-attention layers keep one;
    with tp_size > num_key_value_heads each KV head lives on tp/kv ranks."""
    local_kv = max(1, config.num_key_value_heads // tp_size)
    per_layer = batch * max_seq_len * local_kv * config.head_dim * 2
    return 2 * config.num_full_attention_layers * per_layer


def deltanet_state_bytes(config: QwenConfig, batch: int = 1, tp_size: int = 1) -> int:
    vh = config.linear_num_value_heads // tp_size
    per = vh * config.linear_key_head_dim * config.linear_value_head_dim * 4
    conv = (config.linear_conv_dim // tp_size) * (config.linear_conv_kernel_dim - 1) * 2
    return config.num_linear_attention_layers * batch * (per + conv)


def memory_budget(config: QwenConfig, max_seq_len: int = 2048, num_gpus: int = 1,
                  batch: int = 1, int4_attention: Optional[bool] = None,
                  hbm_bytes: int = B200_HBM_BYTES) -> dict:
    """Per-GPU memory estimate (weights sharded by TP, embeddings replicated,
    lm_head vocab-sharded)."""
    int4_attn = config.attn_quantized if int4_attention is None else int4_attention
    h, inter = config.hidden_size, config.intermediate_size
    g = config.group_size
    n_full, n_lin = config.num_full_attention_layers, config.num_linear_attention_layers
    attn_params = n_full * h * (2 * config.full_attn_q_dim + 2 * config.full_attn_kv_dim
                                + config.full_attn_q_dim)
    lin_params = n_lin * h * (config.linear_conv_dim + 2 * config.linear_attn_value_dim)
    ffn_params = config.num_hidden_layers * 3 * h * inter

    def int4_bytes(p):
        return p // 2 + (p // g) * 2 + (p // g) // 2

    ffn_bytes = int4_bytes(ffn_params)
    attn_bytes = int4_bytes(attn_params + lin_params) if int4_attn else 2 * (attn_params + lin_params)
    embed_bytes = config.vocab_size * h * 2
    lm_head_bytes = config.vocab_size * h * 2
    sharded = ffn_bytes + attn_bytes + lm_head_bytes
    kv = kv_cache_bytes(config, max_seq_len, batch, num_gpus)
    dn = deltanet_state_bytes(config, batch, num_gpus)
    scratch = max_seq_len * h * 4 * 8
    per_gpu = sharded / num_gpus + embed_bytes + kv + dn + scratch
    total = sharded + embed_bytes + (kv + dn) * num_gpus + scratch
    return {
        "model_gb": (sharded + embed_bytes) / 1e9,
        "attn_gb": attn_bytes / 1e9,
        "ffn_int4_gb": ffn_bytes / 1e9,
        "kv_cache_gb_per_gpu": kv / 1e9,
        "deltanet_state_gb_per_gpu": dn / 1e9,
        "scratch_gb": scratch / 1e9,
        "total_gb": total / 1e9,
        "per_gpu_gb": per_gpu / 1e9,
        "fits_per_gpu": per_gpu < hbm_bytes,
        "min_gpus": max(1, int(-(-total // hbm_bytes))),
    }


# ---------------------------------------------------------------------------
# Decoders whose layers are described one by one: mixers made of windowed
# attention and / or a linear recurrence, and a dense feed-forward.
# ---------------------------------------------------------------------------

@dataclass(frozen=True)
class WindowAttentionSpec:
    """Sliding-window attention."""
    heads: int
    kv_heads: int
    dim: int
    rot_dims: int                     # 0: no rotation
    rot_base: float
    scale: float
    window: int                       # 0: unlimited
    vdim: int = 0                     # size of a value head; 0: the values are the keys as projected
    head_norm: bool = False           # Q and K normalised per head (one weight for all heads) or over the whole projection
    keep_first: int = 0               # first tokens that stay visible beyond the window
    softcap: float = 0.0              # scores become softcap * tanh(score / softcap); 0: none
    sink: bool = False                # a learned number per head joins the soft-max's denominator

    @property
    def vd(self) -> int:
        return self.vdim or self.dim

    def check(self, where: str):
        if (self.heads < 1 or self.kv_heads < 1 or self.heads % self.kv_heads or self.rot_dims % 2 or self.rot_dims > self.dim
                or not 1 <= self.dim <= 256 or not 1 <= self.vd <= 256 or self.window < 0 or self.keep_first < 0):
            raise ValueError(f"{where}: unsupported attention sizes {self}")

    def cache_bytes_per_token(self, elem: int) -> int:
        """A K and a V row (head rows padded to 8 elements)."""
        return self.kv_heads * (-(-self.dim // 8) * 8 + -(-self.vd // 8) * 8) * elem


@dataclass(frozen=True)
class SSDSpec:
    """Mamba-2 recurrence: `heads` of size `vdim`, state size `state`, B and C
    shared by the heads of a group, gated RMSNorm in `norm_groups` parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                         # taps of the causal convolution
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def check(self, where: str):
        if self.heads % self.groups or self.inner % self.norm_groups or not 1 <= self.state <= 256 or self.conv < 1:
            raise ValueError(f"{where}: unsupported recurrence sizes {self}")


@dataclass(frozen=True)
class LightningSpec:
    """Linear attention over a state that fades by a constant factor per head and token; every head has its own
    q and k (of size `state`) and v (of size `vdim`)."""
    heads: int
    state: int
    vdim: int
    decay: tuple

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    # no convolution in front of it
    conv, conv_channels = 1, 0

    def check(self, where: str):
        if self.heads < 1 or self.vdim < 1 or not 1 <= self.state <= 256 or len(self.decay) != self.heads \
                or any(not 0.0 <= x <= 1.0 for x in self.decay):
            raise ValueError(f"{where}: unsupported recurrence sizes {self}")


def _cache_bytes(mixers, max_seq_len: int, batch: int, elem: int) -> int:
    return sum(batch * max_seq_len * a.cache_bytes_per_token(elem) for a, _ in mixers if a is not None)


def _state_bytes(mixers, batch: int, elem: int) -> int:
    return sum(batch * (s.heads * s.state * s.vdim * 4 + (s.conv - 1) * s.conv_channels * elem) for _, s in mixers if s is not None)


@dataclass(frozen=True)
class ParallelLayerSpec:
    attention: WindowAttentionSpec
    ssd: SSDSpec
    left_scale: float
    right_scale: float
    ff: int = 0                       # 0: no feed-forward
    weights_of: Optional[int] = None  # layer whose tensors this one uses


@dataclass
class DegedraConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    layers: List[ParallelLayerSpec]
    logit_softcap: float = 0.0        # 0: none

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            l.attention.check(f"layer {i}")
            l.ssd.check(f"layer {i}")
            self.weight_layer(i)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def weight_layer(self, i: int) -> int:
        """Index of the layer whose tensors layer i uses (itself, if it has its own)."""
        seen = set()
        while self.layers[i].weights_of is not None:
            seen.add(i)
            i = self.layers[i].weights_of
            if not 0 <= i < len(self.layers) or i in seen:
                raise ValueError("weights_of does not lead to a layer with tensors")
        return i

    def run_order(self) -> List[int]:
        """Layer of every run of a layer in a step."""
        return list(range(len(self.layers)))

    def run_mixers(self) -> list:
        """(attention or None, recurrence or None) of every run: what it keeps in the cache and the state."""
        return [(l.attention, l.ssd) for l in self.layers]

    def cache_bytes(self, max_seq_len: int, batch: int = 1, elem: int = 2) -> int:
        return _cache_bytes(self.run_mixers(), max_seq_len, batch, elem)

    def state_bytes(self, batch: int = 1, elem: int = 2) -> int:
        return _state_bytes(self.run_mixers(), batch, elem)


def tiny_degedra_config() -> DegedraConfig:
    """Three small layers, the last one sharing the first one's tensors (smoke runs, examples)."""
    a = WindowAttentionSpec(heads=6, kv_heads=2, dim=48, rot_dims=32, rot_base=10000.0, scale=48 ** -0.5, window=40)
    s = SSDSpec(heads=6, vdim=32, state=64, groups=3, conv=4, norm_groups=3)
    l = ParallelLayerSpec(a, s, 0.9, 0.7, 320)
    return DegedraConfig(256, 1000, 1e-6, [l, dataclasses.replace(l, ff=0), dataclasses.replace(l, weights_of=0)], 25.0)


def degedra_config_from_dict(c: dict) -> DegedraConfig:
    layers = []
    for i, e in enumerate(c["layers"]):
        if e.get("type") != "parallel":
            raise ValueError(f"layer {i}: unknown mixer type {e.get('type')!r}")
        m = e["mixer"]
        a, r = m["left"], m["right"]
        if a.get("vdim", a["dim"]) != a["dim"]:
            raise ValueError(f"layer {i}: the values are the projected keys, so vdim must equal dim")
        mlp = e.get("mlp")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        layers.append(ParallelLayerSpec(
            attention=WindowAttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["rot"]["dims"], float(a["rot"]["base"]),
                                          float(a["scale"]), int((a.get("mask") or {}).get("size") or 0)),
            ssd=SSDSpec(r["heads"], r["vdim"], r["state"], r["groups"], r["conv"], r["norm_groups"]),
            left_scale=float(m["left_scale"]), right_scale=float(m["right_scale"]),
            ff=0 if mlp is None else mlp["ff"], weights_of=e.get("weights_of")))
    return DegedraConfig(hidden_size=c["width"], vocab_size=c["vocab"], rms_norm_eps=float(c["norm"]["eps"]),
                         layers=layers, logit_softcap=float(c.get("logit_softcap") or 0.0))


def degedra_config_to_dict(cfg: DegedraConfig) -> dict:
    """The config.json form that `degedra_config_from_dict` reads."""
    layers = []
    for l in cfg.layers:
        a, s = l.attention, l.ssd
        e = {"type": "parallel",
             "mixer": {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "scale": a.scale,
                                "rot": {"base": a.rot_base, "dims": a.rot_dims}, "mask": {"size": a.window}},
                       "right": {"heads": s.heads, "vdim": s.vdim, "state": s.state, "groups": s.groups, "conv": s.conv,
                                 "norm_groups": s.norm_groups},
                       "left_scale": l.left_scale, "right_scale": l.right_scale},
             "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None}
        if l.weights_of is not None:
            e["weights_of"] = l.weights_of
        layers.append(e)
    out = {"architecture": "Degedra", "width": cfg.hidden_size, "vocab": cfg.vocab_size,
           "norm": {"eps": cfg.rms_norm_eps}, "layers": layers}
    if cfg.logit_softcap:
        out["logit_softcap"] = cfg.logit_softcap
    return out


# Vekerax: pre-norm decoder over several residual streams, each layer with one mixer (attention or lightning
# attention), some of the layers run several times with the same weights.

@dataclass(frozen=True)
class StreamLayerSpec:
    """One mixer (a `WindowAttentionSpec` or a `LightningSpec`) and a feed-forward."""
    mixer: object
    ff: int = 0                       # 0: no feed-forward
    act: str = "relu"                 # of the feed-forward's gate

    @property
    def attention(self) -> Optional[WindowAttentionSpec]:
        return self.mixer if isinstance(self.mixer, WindowAttentionSpec) else None

    @property
    def recurrence(self) -> Optional[LightningSpec]:
        return self.mixer if isinstance(self.mixer, LightningSpec) else None


MAX_STREAMS = 16


@dataclass
class VekeraxConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    layers: List[StreamLayerSpec]
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    streams: int = 0                  # residual streams joined by hyper-connections; 0: one stream, plain residual sums
    loop: Optional[tuple] = None      # (start, stop, times): layers start .. stop-1 run `times` times in a row

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            l.mixer.check(f"layer {i}")
        if not 0 <= self.streams <= MAX_STREAMS:
            raise ValueError(f"at most {MAX_STREAMS} residual streams")
        if self.loop is not None:
            a, b, n = self.loop
            if not 0 <= a <= b <= len(self.layers) or n < 0:
                raise ValueError(f"the loop {self.loop} does not fit {len(self.layers)} layers")

    @property
    def num_hidden_layers(self) -> int:
        """Layers with weights (a looped one counts once)."""
        return len(self.layers)

    def run_order(self) -> List[int]:
        """Layer of every run of a layer in a step."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def run_mixers(self) -> list:
        """(attention or None, recurrence or None) of every run: each has a cache or state of its own."""
        return [(self.layers[i].attention, self.layers[i].recurrence) for i in self.run_order()]

    def cache_bytes(self, max_seq_len: int, batch: int = 1, elem: int = 2) -> int:
        return _cache_bytes(self.run_mixers(), max_seq_len, batch, elem)

    def state_bytes(self, batch: int = 1, elem: int = 2) -> int:
        return _state_bytes(self.run_mixers(), batch, elem)


def tiny_vekerax_config() -> VekeraxConfig:
    """Three small layers, two of them run three times, three streams (smoke runs, examples)."""
    a = WindowAttentionSpec(6, 2, 48, 0, 0.0, 48 ** -0.5, 40, vdim=32, head_norm=True, keep_first=3, softcap=20.0, sink=True)
    s = LightningSpec(4, 24, 40, (0.5, 0.9, 0.99, 1.0))
    return VekeraxConfig(256, 1000, 1e-6, [StreamLayerSpec(a, 320), StreamLayerSpec(s, 320), StreamLayerSpec(a)], 2.0, 0.6, 3, (1, 3, 3))


def vekerax_config_from_dict(c: dict) -> VekeraxConfig:
    layers = []
    for i, e in enumerate(c["layers"]):
        m, mlp = e["mixer"], e.get("mlp")
        if e.get("type") == "attention":
            mask = m.get("mask") or {}
            mixer = WindowAttentionSpec(m["heads"], m["kv_heads"], m["dim"], 0, 0.0, float(m["scale"]), int(mask.get("size") or 0),
                                        vdim=m["vdim"], head_norm=True, keep_first=int(mask.get("keep_first") or 0),
                                        softcap=float(m.get("softcap") or 0.0), sink=True)
        elif e.get("type") == "lightning":
            mixer = LightningSpec(m["heads"], m["dim"], m["vdim"], tuple(float(x) for x in m["decay"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {e.get('type')!r}")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        layers.append(StreamLayerSpec(mixer, 0 if mlp is None else mlp["ff"]))
    loop = c.get("loop")
    return VekeraxConfig(hidden_size=c["width"], vocab_size=c["vocab"], rms_norm_eps=float(c["norm"]["eps"]), layers=layers,
                         embedding_scale=float((c.get("embedding") or {}).get("scale", 1.0)),
                         residual_mult=float(c.get("residual_mult", 1.0)), streams=int(c.get("streams") or 0),
                         loop=None if not loop else (loop["start"], loop["stop"], loop["times"]))


def vekerax_config_to_dict(cfg: VekeraxConfig) -> dict:
    """The config.json form that `vekerax_config_from_dict` reads."""
    layers = []
    for l in cfg.layers:
        if l.attention is not None:
            a = l.attention
            e = {"type": "attention", "mixer": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vd, "scale": a.scale}}
            if a.softcap:
                e["mixer"]["softcap"] = a.softcap
            if a.window:
                e["mixer"]["mask"] = {"size": a.window, "keep_first": a.keep_first}
        else:
            r = l.recurrence
            e = {"type": "lightning", "mixer": {"heads": r.heads, "dim": r.state, "vdim": r.vdim, "decay": list(r.decay)}}
        e["mlp"] = {"kind": "dense", "ff": l.ff} if l.ff else None
        layers.append(e)
    out = {"architecture": "Vekerax", "width": cfg.hidden_size, "vocab": cfg.vocab_size, "norm": {"eps": cfg.rms_norm_eps},
           "embedding": {"scale": cfg.embedding_scale}, "residual_mult": cfg.residual_mult, "layers": layers}
    if cfg.streams:
        out["streams"] = cfg.streams
    if cfg.loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), cfg.loop))
    return out


AR_MODES = ("exact", "deferred_ref", "deferred_consistent")


@dataclass(frozen=True)
class EngineConfig:
    """How an engine runs.  `ar_mode`: 'exact' does two all-reduces per layer;
    'deferred_ref' reproduces the reference's deferred attention all-reduce
    (each rank adds only its own attention partial; reference:
    src/runtime/c_dispatch.c:1110-1121); 'deferred_consistent' sends the
    attention partial along with the FFN partial so the ranks' residual streams
    re-converge after every layer with one all-reduce per layer."""
    tp_size: int = 1
    tp_rank: int = 0
    max_seq_len: int = 2048
    max_batch: int = 1
    quant_format: str = "w4a16"
    use_int4_attention: bool = False
    ar_mode: str = "exact"
    use_graph: bool = True
    use_multimem: bool = True
    fused_gemv_ar: bool = True
    # the persistent projection-chain kernel (csrc/chain.cu) in the decode step: 0 off, 1 consecutive INT4
    # projections run as one launch, 2 only the projections that exchange across GPUs use it (one launch each),
    # -1 (default, or B200GRAD_CHAIN unset) = 2 on two to four GPUs, 0 otherwise
    use_chain: int = dataclasses.field(default_factory=lambda: int(os.environ.get("B200GRAD_CHAIN", "-1")))
    # many-row steps under tensor parallelism: 1 = residual stream sequence-parallel between the row-parallel
    # projections (reduce-scatter by token rows + norm + fp16 all-gather in one kernel), 0 = all-reduce + norm
    seq_parallel: int = dataclasses.field(default_factory=lambda: int(os.environ.get("B200GRAD_SEQ_PARALLEL", "1")))
    spec_ngram: int = 3
    spec_max_draft: int = 4
    max_step_rows: int = 0           # rows of a batched-decode / verify step (0: 8 per sequence slot)
    wait_budget_us: int = 2_000_000
    debug_guards: bool = False

    def __post_init__(self):
        if self.ar_mode not in AR_MODES:
            raise ValueError(f"ar_mode must be one of {AR_MODES}")
        if self.quant_format not in ("w4a16", "w8a8", "w4a8"):
            raise ValueError("quant_format must be w4a16, w8a8 or w4a8")

    def replace(self, **kw) -> "EngineConfig":
        return dataclasses.replace(self, **kw)

    @staticmethod
    def from_env(**kw) -> "EngineConfig":
        """Constructor kwargs overridden by B200GRAD_* environment variables."""
        env = os.environ
        if "B200GRAD_AR_MODE" in env:
            kw["ar_mode"] = env["B200GRAD_AR_MODE"]
        if "B200GRAD_GRAPH" in env:
            kw["use_graph"] = env["B200GRAD_GRAPH"] not in ("0", "false", "")
        if "B200GRAD_MULTIMEM" in env:
            kw["use_multimem"] = env["B200GRAD_MULTIMEM"] not in ("0", "false", "")
        if "B200GRAD_DEBUG_GUARDS" in env:
            kw["debug_guards"] = env["B200GRAD_DEBUG_GUARDS"] not in ("0", "false", "")
        return EngineConfig(**kw)
