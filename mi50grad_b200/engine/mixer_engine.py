"""Engine of the decoders whose layers are described one by one, on one GPU: the
post-norm decoder of parallel mixers (Degedra) here, the pre-norm decoder over
residual streams (Vekerax) in `vekerax_engine`, which replaces only what a layer is
made of.

The token-level interface, the row templates, the graph-captured decode step and the
C++ driver are those of `InferenceEngine`; what differs is what the driver is given:
dense bf16 (or, for a model run entirely in 32 bits, fp32) projections fused per
layer, caches and recurrent states of every run of a layer (`MixerStates`), and the
work buffers of the mixer kernels.

Fusions made when weights are loaded (Degedra):
* [q | k | right.in] is one in-projection, so both branches of the mixer come from one
  launch;
* the branches' output projections are one matrix over the concatenation
  [attention | recurrence]; the kernels that produce those columns multiply them by
  left_scale / right_scale before they are rounded;
* gate and up rows are interleaved by 8, so the projection's epilogue forms
  silu(gate) * up.
"""
from __future__ import annotations

import ctypes as C
from types import SimpleNamespace
from typing import Dict, List, Optional, Sequence, Union

import numpy as np
import torch

from ..config import EngineConfig, WindowAttentionSpec
from ..models.mixer_weights import MixerLayerWeights, MixerModelWeights, random_mixer_model
from ..ops import lib as L
from .engine import InferenceEngine
from .state import MixerStates

DTYPES = {"bfloat16": (torch.bfloat16, L.DT_BF16, L.LIN_BF16), "float32": (torch.float32, L.DT_F32, L.LIN_F32)}


def _up8(n: int) -> int:
    return -(-n // 8) * 8


def gemv_outputs_per_cta(n: int, tensor_core: bool, pair: bool = False) -> int:
    """Outputs per CTA of a decode projection with n outputs: as many as leave every SM about one and a half
    CTAs (the tensor-core kernel takes at least 16, the other at least 8, a gate / up pair at least 16)."""
    for r in (32, 16):
        if n >= r * 222:
            return r
    return 16 if tensor_core or pair else 8


class MixerLinear:
    """A dense projection on the GPU: [N][K padded to 8] in the engine's element type."""

    def __init__(self, w: torch.Tensor, kind: int, dtype: torch.dtype, device, pair: bool = False):
        self.N, self.K = w.shape
        self.kind = kind
        self.rpc_few = gemv_outputs_per_cta(self.N, False, pair)         # one or two rows, and fp32
        self.rpc = gemv_outputs_per_cta(self.N, True) if kind == L.LIN_BF16 else self.rpc_few
        self.w = torch.zeros(self.N, _up8(self.K), dtype=dtype, device=device)
        self.w[:, :self.K].copy_(w)

    def desc(self) -> L.LinearDesc:
        d = L.LinearDesc()
        d.kind, d.K, d.N, d.ldw, d.w = self.kind, self.K, self.N, self.w.shape[1], self.w.data_ptr()
        d.L, d.kslice = self.rpc, self.rpc_few
        return d

    def nbytes(self) -> int:
        return self.w.numel() * self.w.element_size()


def fill_attention(m: L.MixLayer, a: WindowAttentionSpec, k: torch.Tensor, v: torch.Tensor, off_q: int, separate_values: bool):
    """Sizes, constants, caches and projection columns [q | k (| v)] of an attention."""
    m.H, m.G, m.d, m.dp, m.rot, m.window = a.heads, a.kv_heads, a.dim, _up8(a.dim), a.rot_dims, a.window
    m.dv, m.vp, m.head_norm, m.keep_first, m.softcap = a.vd, _up8(a.vd), int(a.head_norm), a.keep_first, a.softcap
    m.attn_scale, m.kcache, m.vcache = a.scale, k.data_ptr(), v.data_ptr()
    m.off_q, m.off_k = off_q, off_q + a.heads * a.dim
    m.off_v = m.off_k + a.kv_heads * a.dim if separate_values else -1


def interleave_dense_gate_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[F, K] x 2 -> [2 * F', K] with rows g0..g7 u0..u7 g8.. (F' = F padded to 8 with zero rows)."""
    F, K = gate.shape
    Fp = _up8(F)
    both = torch.zeros(Fp // 8, 2, 8, K, dtype=gate.dtype, device=gate.device)
    for j, w in enumerate((gate, up)):
        p = torch.zeros(Fp, K, dtype=w.dtype, device=w.device)
        p[:F] = w
        both[:, j] = p.reshape(Fp // 8, 8, K)
    return both.reshape(2 * Fp, K)


class MixerLayer:
    """Device weights of one layer (shared by layers that use another's tensors)."""

    def __init__(self, eng: "MixerEngine", lw: MixerLayerWeights, layer_idx: int):
        dev, f32 = eng.device, eng._f32
        t = lambda w: w.to(device=dev, dtype=eng.dtype)
        lin = lambda w, pair=False: MixerLinear(w, eng.lin_kind, eng.dtype, dev, pair)
        self.in_proj = lin(torch.cat([t(lw.q), t(lw.k), t(lw.ssd_in)], 0))
        self.out_proj = lin(torch.cat([t(lw.attn_o), t(lw.ssd_o)], 1))
        self.gate_up = self.down = None
        if lw.gate is not None:
            self.gate_up = lin(interleave_dense_gate_up(t(lw.gate), t(lw.up)), True)
            self.down = lin(t(lw.down))
        self.norm1, self.norm2 = f32(lw.norm1), None if lw.norm2 is None else f32(lw.norm2)
        self.q_norm, self.k_norm = f32(lw.q_norm), f32(lw.k_norm)
        self.conv, self.conv_b = f32(lw.conv), f32(lw.conv_b)
        self.dt_bias, self.A_log, self.D, self.ssd_norm = f32(lw.dt_bias), f32(lw.A_log), f32(lw.D), f32(lw.ssd_norm)

    def linears(self) -> List[MixerLinear]:
        return [l for l in (self.in_proj, self.out_proj, self.gate_up, self.down) if l is not None]


class MixerEngine(InferenceEngine):
    """`layer_type`, `weights_type` and the methods `_mix_layer`, `_layer_desc`, `_extend_model` are what an
    architecture of this kind replaces."""
    layer_type = MixerLayer
    weights_type = MixerLayerWeights

    def __init__(self, config, device_id: int = 0, max_seq_len: int = 2048, dtype: str = "bfloat16",
                 engine_config: Optional[EngineConfig] = None, max_batch: int = 1):
        if dtype not in DTYPES:
            raise ValueError(f"dtype must be one of {sorted(DTYPES)}")
        if not torch.cuda.is_available():
            raise RuntimeError(f"{type(self).__name__} needs a CUDA device")
        self.dtype_name = dtype
        self.dtype, self.dt, self.lin_kind = DTYPES[dtype]
        self._init_common(config, device_id, max_seq_len, 1, 0, engine_config, None, max_batch)
        self.spec = SimpleNamespace(vocab=(0, config.vocab_size), vocab_local=config.vocab_size)
        self.runs = config.run_order()               # layer of every run of a layer in a step
        if not self.runs:
            raise ValueError("the model runs no layer")
        self.states = MixerStates(config, max_seq_len, max_batch, self.device, self.dtype)
        self.use_tc_prefill = True       # many rows have a path of their own in both element types
        self._shared: Dict[int, MixerLayer] = {}
        self._rope: Dict[tuple, tuple] = {}

    # ------------------------------------------------------------------ weights
    def _f32(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=torch.float32).contiguous()

    def _weight_layer(self, i: int) -> int:
        return self.config.weight_layer(i)

    def load_layer_weights(self, layer_idx: int, lw: Union[MixerLayerWeights, dict]):
        """A layer that uses another layer's tensors gets that layer's device weights, whichever of them is
        loaded first."""
        if isinstance(lw, dict):
            lw = self.weights_type(**lw)
        j = self._weight_layer(layer_idx)
        if j == layer_idx or j not in self._shared:
            self._shared[j] = self.layer_type(self, lw, layer_idx)
            for i in range(len(self.layers)):
                if self.layers[i] is not None and self._weight_layer(i) == j:
                    self.layers[i] = self._shared[j]
        self.layers[layer_idx] = self._shared[j]
        self._drop_driver()

    def load_final_norm(self, w: torch.Tensor):
        self.final_norm = self._f32(torch.as_tensor(w))
        self._drop_driver()

    def load_lm_head(self, w: torch.Tensor):
        self.lm_head = MixerLinear(torch.as_tensor(w), self.lin_kind, self.dtype, self.device)
        self._drop_driver()

    def load_embedding(self, w: torch.Tensor):
        self.embed = torch.as_tensor(w).to(device=self.device, dtype=self.dtype).contiguous()
        self._drop_driver()

    def load_model(self, mw: MixerModelWeights):
        for i, lw in enumerate(mw.layers):
            if self._weight_layer(i) == i:
                self.load_layer_weights(i, lw)
        for i, lw in enumerate(mw.layers):
            if self._weight_layer(i) != i:
                self.load_layer_weights(i, lw)
        self.load_embedding(mw.embed)
        self.load_lm_head(mw.head)
        self.load_final_norm(mw.final_norm)

    def init_random(self, seed: int = 0, **_):
        self.load_model(random_mixer_model(self.config, seed, self.device, self.dtype))

    def weight_bytes(self) -> int:
        """Bytes one decode step streams (a layer counts every time it runs)."""
        return sum(l.nbytes() for i in self.runs for l in self.layers[i].linears()) + self.lm_head.nbytes()

    def _rope_tables(self, base: float, rot: int):
        key = (base, rot)
        if key not in self._rope:
            f = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
            ang = torch.arange(self.max_seq_len, dtype=torch.float64)[:, None] * f[None, :]
            self._rope[key] = (self._f32(torch.cos(ang)), self._f32(torch.sin(ang)))
        return self._rope[key]

    # ------------------------------------------------------------------ driver
    def _mix_layer(self, run: int) -> L.MixLayer:
        """Sizes, constants and pointers of run `run` of a layer for the mixer kernels."""
        i = self.runs[run]
        l, dl, st = self.config.layers[i], self.layers[i], self.states
        a, s = l.attention, l.ssd
        m = L.MixLayer()
        fill_attention(m, a, st.k[run], st.v[run], 0, False)
        m.left_scale, m.right_scale, m.eps = l.left_scale, l.right_scale, self.config.rms_norm_eps
        m.q_norm, m.k_norm = dl.q_norm.data_ptr(), dl.k_norm.data_ptr()
        cos, sin = self._rope_tables(a.rot_base, a.rot_dims)
        m.cos_tab, m.sin_tab = cos.data_ptr(), sin.data_ptr()
        m.heads, m.P, m.N, m.groups, m.ngroups, m.taps = s.heads, s.vdim, s.state, s.groups, s.norm_groups, s.conv
        m.conv_w, m.conv_b, m.dt_bias = dl.conv.data_ptr(), dl.conv_b.data_ptr(), dl.dt_bias.data_ptr()
        m.A_log, m.D, m.norm_w = dl.A_log.data_ptr(), dl.D.data_ptr(), dl.ssd_norm.data_ptr()
        m.state, m.conv_state = st.S[run].data_ptr(), st.conv[run].data_ptr()
        m.off_z = m.off_k + a.kv_heads * a.dim
        m.off_x = m.off_z + s.inner
        m.off_dt = m.off_x + s.conv_channels
        m.rx, m.rB, m.rC = 0, s.inner, s.inner + s.groups * s.state
        m.gate, m.out_col = L.REC_GATE_SILU_NORM, a.heads * a.dim
        m.max_seq = self.max_seq_len
        return m

    def _layer_desc(self, d: L.MixerLayerDesc, run: int):
        """What the driver needs beyond the mixer's block and the projections."""
        ly = self.layers[self.runs[run]]
        d.kind, d.norm1 = L.MIX_PARALLEL, ly.norm1.data_ptr()
        if ly.down is not None:
            d.norm2 = ly.norm2.data_ptr()

    def _extend_model(self, x: L.MixerModelDesc, alloc):
        """Architecture-wide parts of the driver's model description."""

    def _ensure_driver(self):
        if self._driver is not None:
            return
        if any(l is None for l in self.layers) or self.embed is None or self.lm_head is None or self.final_norm is None:
            raise RuntimeError("weights are not fully loaded")
        cfg, R, T = self.config, self.max_rows, self.dtype
        H, P = cfg.hidden_size, min(512, self.max_seq_len)
        self.max_prefill = P
        runs, n_runs = [self.layers[i] for i in self.runs], len(self.runs)
        alloc = self._work_allocator()
        f32 = lambda *s: alloc(s, torch.float32)
        i32 = lambda *s: alloc(s, torch.int32)
        elt = lambda *s: alloc(s, T)
        mix = [self._mix_layer(i) for i in range(n_runs)]
        att, rec = [m for m in mix if m.H], [m for m in mix if m.heads]
        b = self.buf = {}
        ld_x = _up8(H)
        b["ld_proj"] = _up8(max(ly.in_proj.N for ly in runs))
        b["ld_attn"] = _up8(max(ly.out_proj.K for ly in runs))
        ld_act = _up8(max([ly.down.K for ly in runs if ly.down is not None] + [8]))
        b["ld_logits"] = -(-cfg.vocab_size // 4) * 4
        b["h"], b["h_tmp"], b["m"], b["xn"] = f32(R, H), f32(R, H), f32(R, H), elt(R, ld_x)
        b["proj"], b["attn_out"], b["act"] = elt(R, b["ld_proj"]), elt(R, b["ld_attn"]), elt(R, ld_act)
        b["logits"] = f32(R, b["ld_logits"])
        self.np = -(-H // 8)                                   # one partial sum per CTA of at least 8 outputs
        b["ss"] = f32(R, self.np)
        M_PLANES = 4                                           # splits over K of a many-row output projection
        b["p_h"], b["p_m"], b["p_xn"] = f32(P, H), f32(M_PLANES, P, H), elt(P, ld_x)
        b["p_proj"], b["p_attn"], b["p_act"] = elt(P, b["ld_proj"]), elt(P, b["ld_attn"]), elt(P, ld_act)
        M = max(P, R)
        b["qbuf"] = elt(M, max([m.H * m.dp for m in att] + [8]))
        channels = [s.conv_channels for _, s in cfg.run_mixers() if s is not None]
        ld_xbc, ld_u, ld_dt = _up8(max(channels + [8])), _up8(max([m.heads * m.P for m in rec] + [8])), max([m.heads for m in rec] + [1])
        b["xbc"], b["ubuf"], b["dtb"] = elt(M, ld_xbc), f32(M, ld_u), f32(M, ld_dt)
        # cache slices per decode-attention row: as many as the widest window can use
        widest = max([min(m.window + m.keep_first if m.window else self.max_seq_len, self.max_seq_len) for m in att] + [1])
        self.attn_splits = max(1, min(32, -(-widest // 64)))
        SR = max(R, self.max_batch)                            # rows the split-attention scratch holds
        b["attn_scratch"] = f32(max([self.lib.b2_window_attn_scratch(m.H, m.G, max(m.dp, m.vp), SR, self.attn_splits) for m in att] + [8]))
        b["attn_counters"] = i32(max([self.lib.b2_window_attn_units(m.H, m.G, SR) for m in att] + [0]) + 8)
        b["ssd_counters"] = i32(max([self.lib.b2_ssd_units(C.byref(m), SR) for m in rec] + [0]) + 8)
        if self.dt == L.DT_BF16 and rec:
            b["chunk_state"] = f32(max(self.lib.b2_ssd_chunk_state_floats(C.byref(m), P) for m in rec))
            b["chunk_prev"] = alloc((max(self.lib.b2_ssd_chunk_prev_bytes(C.byref(m), P) for m in rec),), torch.uint8)
            b["chunk_decay"] = f32(-(-P // 64) * ld_dt)
        self.argmax_blocks = max(1, min(64, cfg.vocab_size // 2048))
        b["argmax_scratch"], b["argmax_counters"] = f32(R * self.argmax_blocks * 2), i32(R + 8)
        b["rows"], b["rows_tmpl"], b["p_rows"], b["p_rows_tmpl"] = i32(R, 6), i32(R, 6), i32(P, 6), i32(P, 6)
        b["row_tokens"] = torch.full((R,), -1, dtype=torch.int32, device=self.device)
        b["p_row_tokens"] = torch.full((P,), -1, dtype=torch.int32, device=self.device)
        b["seq_rows"] = i32(self.max_batch + 1 + R)
        b["out_tokens"], b["p_out_tokens"], b["tc_status"] = i32(R), i32(P), i32(4)
        # rows of a many-row step that can have logits: what the caller asked for, or 64 MB of them
        want = self.ecfg.max_step_rows or max(8 * self.max_batch, (64 << 20) // (4 * b["ld_logits"]))
        self.step_rows = min(P, max(8, want))
        b["p_logits"] = f32(self.step_rows, b["ld_logits"])
        b["p_argmax_scratch"], b["p_argmax_counters"] = f32(self.step_rows * self.argmax_blocks * 2), i32(self.step_rows + 8)

        x = L.MixerModelDesc()
        x.final_norm, x.softcap, x.dt = self.final_norm.data_ptr(), getattr(cfg, "logit_softcap", 0.0), self.dt
        x.ss_np, x.ld_x, x.ld_xbc, x.ld_dt, x.ld_u, x.ld_act, x.scratch_rows = self.np, ld_x, ld_xbc, ld_dt, ld_u, ld_act, SR
        x.m_planes = M_PLANES
        for k in ("m", "p_m", "qbuf", "xbc", "dtb", "ubuf", "attn_scratch", "attn_counters", "ssd_counters", "chunk_state",
                  "chunk_prev", "chunk_decay"):
            if k in b:
                setattr(x, k, b[k].data_ptr())
        self._extend_model(x, alloc)
        descs = (L.MixerLayerDesc * n_runs)()
        for r, ly in enumerate(runs):
            d = descs[r]
            d.mix, d.in_proj, d.out_proj = mix[r], ly.in_proj.desc(), ly.out_proj.desc()
            d.gate_up.kind = d.down.kind = L.LIN_NONE
            if ly.down is not None:
                d.gate_up, d.down = ly.gate_up.desc(), ly.down.desc()
            self._layer_desc(d, r)
        x.layers = C.addressof(descs)
        m = L.ModelDesc()
        m.n_layers, m.H, m.vocab, m.vocab_local = n_runs, H, cfg.vocab_size, cfg.vocab_size
        m.max_seq, m.max_rows, m.max_prefill, m.p_logit_rows = self.max_seq_len, R, P, self.step_rows
        m.attn_splits, m.argmax_blocks, m.n_seqs_max, m.eps = self.attn_splits, self.argmax_blocks, self.max_batch, cfg.rms_norm_eps
        m.embed, m.lm_head = self.embed.data_ptr(), self.lm_head.desc()
        m.ld_proj, m.ld_attn, m.ld_logits = b["ld_proj"], b["ld_attn"], b["ld_logits"]
        for k in ("h", "h_tmp", "xn", "proj", "attn_out", "act", "logits", "ss", "argmax_scratch", "argmax_counters", "rows",
                  "rows_tmpl", "row_tokens", "seq_rows", "out_tokens", "p_h", "p_xn", "p_proj", "p_attn", "p_act", "p_rows",
                  "p_rows_tmpl", "p_row_tokens", "p_out_tokens", "p_logits", "p_argmax_scratch", "p_argmax_counters", "tc_status"):
            setattr(m, k, b[k].data_ptr())
        m.seqs, m.comm = self.states.seqs.data_ptr(), L.null_comm()
        m.mixer = C.addressof(x)
        self._model_desc = (m, x, descs)
        self._driver = self.lib.b2_driver_create(C.byref(m), None)
        self._graph_key = self._tmpl_key = self._ptmpl_key = None
        self._stream = torch.cuda.Stream(device=self.device)

    def check_status(self):
        """Raise if a tensor-core GEMM gave up on one of its bounded waits."""
        if self._driver is not None and int(self.buf["tc_status"][0].item()):
            self.buf["tc_status"].zero_()
            raise RuntimeError("a bounded barrier wait of the tensor-core GEMM expired")

    # ------------------------------------------------------------------ token-level API
    def prefill_tokens(self, tokens: Sequence[int], seq: int = 0) -> int:
        tokens = list(tokens)
        self._ensure_driver()
        if len(tokens) <= self.max_rows:
            n = len(tokens)
            tok = self.step_tokens(tokens, seq)[n - 1]
            if n > 1:
                self.buf["logits"][0].copy_(self.buf["logits"][n - 1])
                self.buf["h"][0].copy_(self.buf["h"][n - 1])
            self.states.seqs[seq, 1] = tok
            return int(tok.item())
        return self.prefill_tokens_tc(tokens, seq)

    def prefill_tokens_tc(self, tokens: Sequence[int], seq: int = 0) -> int:
        """Prompt in launches of max_prefill rows; the last one also computes the logits of its last row
        (row 0 of the decode step's logits) and their arg-max."""
        self._ensure_driver()
        tokens = list(tokens)
        for i in range(0, len(tokens), self.max_prefill):
            chunk = tokens[i:i + self.max_prefill]
            n = len(chunk)
            last = i + n == len(tokens)
            self.buf["p_row_tokens"][:n].copy_(torch.tensor(chunk, dtype=torch.int32).to(self.device))
            self._prefill_rows(n, seq, L.STEP_EMBED_TOKENS | ((L.STEP_HEAD_LAST | L.STEP_ARGMAX) if last else 0))
        self.buf["h"][:1].copy_(self.buf["p_h"][n - 1:n])
        self.states.seqs[seq, 1] = self.buf["out_tokens"][0]
        return int(self.buf["out_tokens"][0].item())

    def spec_step(self, *args, **kwargs):
        raise NotImplementedError("draft verification is not available for this architecture (windowed attention and "
                                  "the recurrence take consecutive tokens only)")

    # ------------------------------------------------------------------ embedding-in API
    def forward_embeddings(self, embs, seq: int = 0, commit: bool = True) -> torch.Tensor:
        self._ensure_driver()
        e = self._as_dev(embs).reshape(-1, self.config.hidden_size)
        n = e.shape[0]
        if not 1 <= n <= self.max_rows:
            raise ValueError(f"1..{self.max_rows} rows")
        self._template_chain(seq, n)
        self.buf["h"][:n].copy_(e)
        self._run(n, 1, 0 if commit else L.STEP_NO_COMMIT_DELTA)
        if commit:
            self.states.seqs[seq, 0] += n
        return self.buf["xn"][:n, :self.config.hidden_size]

    def forward_embeddings_tree(self, embs, parents, seq: int = 0):
        return self.spec_step()

    def prefill_step(self, token_embeddings, seq: int = 0):
        e = self._as_dev(token_embeddings).reshape(-1, self.config.hidden_size).contiguous()
        self._ensure_driver()
        for i in range(0, e.shape[0], self.max_prefill):
            n = min(self.max_prefill, e.shape[0] - i)
            self.buf["p_h"][:n].copy_(e[i:i + n])
            self._prefill_rows(n, seq, 0)
        self.buf["h"][:1].copy_(self.buf["p_h"][n - 1:n])
        out = self.buf["p_xn"][n - 1, :self.config.hidden_size]
        return out.float().cpu().numpy() if isinstance(token_embeddings, np.ndarray) else out.clone()

    def decode_step(self, token_embedding, position: Optional[int] = None, seq: int = 0):
        if position is not None and position != self.states.length(seq):
            raise ValueError("a recurrent state cannot be moved to another position")
        out = self.forward_embeddings(token_embedding, seq)[0]
        return out.float().cpu().numpy() if isinstance(token_embedding, np.ndarray) else out.clone()

    def decode_step_batch(self, token_embeddings, batch_size: Optional[int] = None, position: Optional[int] = None, seq: int = 0):
        if position is not None and position != self.states.length(seq):
            raise ValueError("a recurrent state cannot be moved to another position")
        e = self._as_dev(token_embeddings).reshape(-1, self.config.hidden_size)
        out = self.forward_embeddings(e if batch_size is None else e[:batch_size], seq)
        return out.float().cpu().numpy() if isinstance(token_embeddings, np.ndarray) else out.clone()

    def compute_logits(self, hidden=None) -> torch.Tensor:
        """Logits of a final-normed hidden state; None = the last step's."""
        self._ensure_driver()
        if hidden is None:
            out = self.buf["logits"][0, :self.config.vocab_size]
            return out.clone()
        from ..ops import kernels as K
        x = self._as_dev(hidden).reshape(1, -1).to(self.dtype)
        out = torch.empty(1, self.config.vocab_size, dtype=torch.float32, device=self.device)
        K.gemv_dense(self.lm_head, x, out, mode=L.DG_STORE_F32, softcap=getattr(self.config, "logit_softcap", 0.0))
        return out[0].cpu().numpy() if isinstance(hidden, np.ndarray) else out[0]
