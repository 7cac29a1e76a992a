"""Engine of the Vekerax decoder on one GPU: pre-norm layers of one mixer each
(attention with kept first tokens, capped scores and a sink, or lightning attention),
several residual streams joined by hyper-connections, and layers that run several
times.  Everything but the content of a layer is `MixerEngine`'s.

Fusions made when weights are loaded:
* [q | k | v] of an attention and [q | k | v | g] of a lightning attention are one
  in-projection; its epilogue applies the lightning's SiLU to q, k and v;
* gate and up rows are interleaved by 8, so the projection's epilogue forms
  relu(gate) * up;
* the residual multiplier is folded into the streams' output weights, and what joins
  two sublayers (the mixing of the streams, the first one's output weights, the second
  one's input weights) is one small array.
"""
from __future__ import annotations

import math

import torch

from ..models.vekerax_weights import VekeraxLayerWeights, random_vekerax_model
from ..ops import lib as L
from .mixer_engine import MixerEngine, MixerLinear, fill_attention, interleave_dense_gate_up

# logarithm of a decay of zero: its powers vanish in fp32 and differences of its multiples stay finite
LOG_ZERO = -200.0


class VekeraxLayer:
    """Device weights of one layer."""

    def __init__(self, eng: "VekeraxEngine", lw: VekeraxLayerWeights, layer_idx: int):
        dev, f32 = eng.device, eng._f32
        spec = eng.config.layers[layer_idx]
        t = lambda w: w.to(device=dev, dtype=eng.dtype)
        lin = lambda w, pair=False: MixerLinear(w, eng.lin_kind, eng.dtype, dev, pair)
        self.act_cols = 0
        if spec.attention is not None:
            self.in_proj = lin(torch.cat([t(lw.q), t(lw.k), t(lw.v)], 0))
            self.q_norm, self.k_norm, self.sink = f32(lw.q_norm), f32(lw.k_norm), f32(lw.sink)
        else:
            r = spec.recurrence
            self.in_proj = lin(torch.cat([t(lw.q), t(lw.k), t(lw.v), t(lw.g)], 0))
            self.act_cols = r.heads * (2 * r.state + r.vdim)
            self.out_norm = f32(lw.out_norm)
            self.decay = f32(torch.tensor(r.decay, dtype=torch.float64))
            self.log_decay = f32(torch.tensor([math.log(x) if x > 0 else LOG_ZERO for x in r.decay], dtype=torch.float64))
        self.out_proj = lin(t(lw.o))
        self.gate_up = self.down = self.norm2 = None
        self.norm1 = f32(lw.norm1)
        if spec.ff:
            self.gate_up = lin(interleave_dense_gate_up(t(lw.gate), t(lw.up)), True)
            self.down = lin(t(lw.down))
            self.norm2 = f32(lw.norm2)
        one = torch.ones(1)
        hc = lambda q: [(one if w is None else w.float().cpu()) for w in
                        (getattr(lw, f"hc{q}_in"), getattr(lw, f"hc{q}_out"), getattr(lw, f"hc{q}_mix"))]
        self.hc1, self.hc2 = hc(1), hc(2)            # (in, out, mix); without streams all ones of size one

    def linears(self):
        return [l for l in (self.in_proj, self.out_proj, self.gate_up, self.down) if l is not None]


class VekeraxEngine(MixerEngine):
    layer_type = VekeraxLayer
    weights_type = VekeraxLayerWeights

    def _weight_layer(self, i: int) -> int:
        return i

    def init_random(self, seed: int = 0, **_):
        self.load_model(random_vekerax_model(self.config, seed, self.device, self.dtype))

    # the output head is the embedding table: one device copy serves both
    def load_lm_head(self, w: torch.Tensor):
        super().load_lm_head(w)
        self.embed = self.lm_head.w

    def load_embedding(self, w: torch.Tensor):
        self.load_lm_head(w)

    # ------------------------------------------------------------------ driver
    def _mix_layer(self, run: int) -> L.MixLayer:
        i = self.runs[run]
        l, dl, st = self.config.layers[i], self.layers[i], self.states
        m = L.MixLayer()
        m.left_scale = m.right_scale = 1.0
        m.eps, m.max_seq, m.exact_weights = self.config.rms_norm_eps, self.max_seq_len, 1
        if l.attention is not None:
            fill_attention(m, l.attention, st.k[run], st.v[run], 0, True)
            m.q_norm, m.k_norm, m.sink = dl.q_norm.data_ptr(), dl.k_norm.data_ptr(), dl.sink.data_ptr()
            return m
        r = l.recurrence
        m.heads, m.P, m.N, m.groups, m.ngroups, m.taps = r.heads, r.vdim, r.state, r.heads, 1, 1
        m.decay, m.log_decay, m.norm_w = dl.decay.data_ptr(), dl.log_decay.data_ptr(), dl.out_norm.data_ptr()
        m.state, m.gate = st.S[run].data_ptr(), L.REC_NORM_SIGMOID
        m.rC, m.rB, m.rx = 0, r.heads * r.state, 2 * r.heads * r.state          # q, k, v
        m.off_z = m.rx + r.inner
        return m

    def _coef(self, hc, into) -> int:
        """Device array mix | out | in for the step from one sublayer (None: the embedding) to the next (None:
        the sum of the streams in front of the final norm)."""
        n = max(1, self.config.streams)
        ones = torch.ones(n)
        _, out, mix = hc if hc is not None else (None, torch.zeros(n), torch.eye(n))
        c = torch.cat([mix.reshape(-1), self.config.residual_mult * out, ones if into is None else into[0]])
        self._coefs.append(self._f32(c))
        return self._coefs[-1].data_ptr()

    def _layer_desc(self, d: L.MixerLayerDesc, run: int):
        layers = [self.layers[i] for i in self.runs]
        ly = layers[run]
        spec = self.config.layers[self.runs[run]]
        nxt = layers[run + 1].hc1 if run + 1 < len(layers) else None
        d.kind = L.MIX_ATTENTION if spec.attention is not None else L.MIX_RECURRENCE
        d.act, d.act_cols = {"silu": L.ACT_SILU, "relu": L.ACT_RELU}[spec.act], ly.act_cols
        d.norm1 = ly.norm1.data_ptr()
        d.hc1 = self._coef(ly.hc1, ly.hc2 if spec.ff else nxt)
        if spec.ff:
            d.norm2 = ly.norm2.data_ptr()
            d.hc2 = self._coef(ly.hc2, nxt)

    def _extend_model(self, x: L.MixerModelDesc, alloc):
        self._coefs = []
        b, H, n = self.buf, self.config.hidden_size, max(1, self.config.streams)
        b["sx"], b["p_sx"] = alloc((self.max_rows, n, H), torch.float32), alloc((self.max_prefill, n, H), torch.float32)
        b["su"] = alloc((self.max_rows, H), torch.float32)
        x.streams, x.ld_embed, x.embed_scale = n, self.embed.stride(0), self.config.embedding_scale
        x.hc0 = self._coef(None, self.layers[self.runs[0]].hc1)
        x.sx, x.p_sx, x.su = b["sx"].data_ptr(), b["p_sx"].data_ptr(), b["su"].data_ptr()
