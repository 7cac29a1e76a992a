"""Small Vekerax configurations and random weights for the tests."""
import torch

from mi50grad_b200.config import (LightningSpec, StreamLayerSpec, VekeraxConfig, WindowAttentionSpec, tiny_vekerax_config,
                                  vekerax_config_to_dict)
from mi50grad_b200.models.vekerax_weights import named_tensors, random_vekerax_model

from vekerax_oracle import Oracle


def A(heads, kv, dim, vdim, window, keep=0, cap=0.0, scale=None):
    return WindowAttentionSpec(heads, kv, dim, 0, 0.0, dim ** -0.5 if scale is None else scale, window, vdim=vdim, head_norm=True,
                               keep_first=keep, softcap=cap, sink=True)


def R(heads, dim, vdim, *decay):
    return LightningSpec(heads, dim, vdim, tuple(decay) or tuple(1.0 - 0.4 ** (1 + i) for i in range(heads)))


def layer(mixer, ff=0):
    return StreamLayerSpec(mixer, ff)


def mixed_config():
    """Layers of different sizes: value heads larger and smaller than key heads, padded head sizes, 12 queries
    per key head, more kept tokens than the window holds, a decay of zero and of one, layers without
    feed-forward, no cap, three streams, a loop in the middle."""
    return VekeraxConfig(hidden_size=168, vocab_size=301, rms_norm_eps=2e-5, embedding_scale=4.0, residual_mult=0.7, streams=3, loop=(1, 4, 2),
                         layers=[layer(R(5, 17, 33, 0.3, 1.0, 0.0, 0.97, 0.9), 200), layer(A(6, 2, 40, 24, 37, 5, 9.0, 0.35), 76),
                                 layer(A(12, 1, 32, 72, 9, 21, 50.0)), layer(R(2, 130, 24)), layer(A(3, 3, 100, 100, 150, 1), 64)])


def odd_width_config():
    """A width that is no multiple of four, a single stream, the loop at the end, unlimited attention."""
    return VekeraxConfig(hidden_size=90, vocab_size=77, rms_norm_eps=1e-6, embedding_scale=1.5, residual_mult=1.0, streams=1, loop=(0, 2, 3),
                         layers=[layer(A(2, 2, 24, 18, 0, 0, 6.0), 33), layer(R(3, 9, 10), 50)])


def plain_config(window=48, keep=4):
    """Powers of two everywhere (the vectorised paths), several 64-wide column blocks, four streams, no loop."""
    return VekeraxConfig(hidden_size=256, vocab_size=640, rms_norm_eps=1e-5, embedding_scale=8.0, residual_mult=0.6, streams=4,
                         layers=[layer(A(4, 2, 128, 128, window, keep, 20.0), 512), layer(R(4, 64, 128, 0.6, 0.95, 0.99, 0.999), 256),
                                 layer(A(8, 2, 64, 64, 2 * window, 2 * keep, 15.0), 256)])


def bare_config():
    """No hyper-connections (plain residual sums), lightning only at both ends, a loop that runs once."""
    return VekeraxConfig(hidden_size=72, vocab_size=50, rms_norm_eps=1e-5, residual_mult=0.5, loop=(1, 2, 1),
                         layers=[layer(R(1, 8, 200), 40), layer(A(5, 1, 8, 16, 20, 3, 4.0), 24), layer(R(6, 16, 16))])


def many_streams_config():
    """More streams than the unrolled forms have."""
    return VekeraxConfig(hidden_size=64, vocab_size=90, rms_norm_eps=1e-5, embedding_scale=3.5, residual_mult=0.4, streams=6, loop=(0, 1, 2),
                         layers=[layer(A(4, 4, 16, 32, 12, 2, 8.0), 48), layer(R(2, 32, 64), 40)])


CONFIGS = {"mixed": mixed_config, "odd_width": odd_width_config, "plain": plain_config, "bare": bare_config,
           "many_streams": many_streams_config, "tiny": tiny_vekerax_config}


def model(name, seed=0, **kw):
    cfg = CONFIGS[name](**kw)
    return cfg, random_vekerax_model(cfg, seed)


def oracle(mw, dtype=torch.float64):
    return Oracle(vekerax_config_to_dict(mw.config), named_tensors(mw), dtype)
