"""Per-sequence device state: KV cache, Gated DeltaNet state, lengths.

The reference keeps a contiguous fp16 KV cache for the full-attention layers
with ONE shared length for all sequences (reference: src/inference/engine.py:79-290,
:94) and an fp32 recurrent state plus fp16 conv history per DeltaNet layer
(reference: src/inference/engine.py:293-369).  Here every sequence slot has its
own length, kept in device memory so captured graphs can read it, and the whole
position-dependent state of a slot can be snapshotted and restored -- which is
what speculative rollback and recovery need and what the reference cannot do
for its DeltaNet layers (reference: src/inference/tp_engine.py:1673-1687).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from ..config import QwenConfig
from ..parallel.sharding import ShardSpec

DN_COLS = 32


class KVCache:
    """[full_layers][batch][max_seq][local_kv_heads][head_dim] fp16, K and V."""

    def __init__(self, cfg: QwenConfig, spec: ShardSpec, max_seq_len: int, max_batch: int, device):
        self.layers = cfg.full_attention_layer_indices()
        self.index = {li: i for i, li in enumerate(self.layers)}
        shape = (len(self.layers), max_batch, max_seq_len, spec.n_kv, cfg.head_dim)
        self.k = torch.zeros(shape, dtype=torch.float16, device=device)
        self.v = torch.zeros(shape, dtype=torch.float16, device=device)
        self.max_seq_len = max_seq_len

    def layer_k(self, layer_idx: int) -> torch.Tensor:
        return self.k[self.index[layer_idx]]

    def layer_v(self, layer_idx: int) -> torch.Tensor:
        return self.v[self.index[layer_idx]]

    def nbytes(self) -> int:
        return 2 * self.k.numel() * 2


class DeltaNetState:
    """fp32 state [lin_layers][batch][v_heads][dk][dv]; fp16 conv history stored
    per consuming CTA: [lin_layers][batch][v_heads][dv/32][2*dk+32][3]."""

    def __init__(self, cfg: QwenConfig, spec: ShardSpec, max_batch: int, device):
        self.layers = cfg.linear_attention_layer_indices()
        self.index = {li: i for i, li in enumerate(self.layers)}
        dk, dv = cfg.linear_key_head_dim, cfg.linear_value_head_dim
        self.nch = 2 * dk + DN_COLS
        self.S = torch.zeros(len(self.layers), max_batch, spec.n_la_v, dk, dv, dtype=torch.float32,
                             device=device)
        self.conv = torch.zeros(len(self.layers), max_batch, spec.n_la_v, dv // DN_COLS, self.nch, 3,
                                dtype=torch.float16, device=device)

    def layer_S(self, layer_idx: int) -> torch.Tensor:
        return self.S[self.index[layer_idx]]

    def layer_conv(self, layer_idx: int) -> torch.Tensor:
        return self.conv[self.index[layer_idx]]

    def nbytes(self) -> int:
        return self.S.numel() * 4 + self.conv.numel() * 2


@dataclass
class SequenceSnapshot:
    """Device copy of everything position-dependent for one sequence slot."""
    seq: int
    length: int
    token: int
    k: Optional[torch.Tensor]
    v: Optional[torch.Tensor]
    S: torch.Tensor
    conv: torch.Tensor


class SlotStates:
    """Sequence slots: the device array `seqs` of {len, token, pad, pad} the kernels
    read, and which slots are handed out."""

    def __init__(self, max_batch: int, device):
        self.seqs = torch.zeros(max_batch, 4, dtype=torch.int32, device=device)
        self.max_batch = max_batch
        self._free = list(range(max_batch))

    def acquire(self) -> int:
        """A free slot, empty."""
        if not self._free:
            raise RuntimeError(f"all {self.max_batch} sequence slots are in use")
        seq = self._free.pop(0)
        self.reset(seq)
        return seq

    def release(self, seq: int):
        """Give a slot back."""
        if seq in self._free or not 0 <= seq < self.max_batch:
            raise ValueError(f"slot {seq} is not in use")
        self._free.insert(0, seq)

    def reset(self, seq: Optional[int] = None):
        raise NotImplementedError

    def lengths(self) -> List[int]:
        return self.seqs[:, 0].tolist()

    def length(self, seq: int = 0) -> int:
        return int(self.seqs[seq, 0].item())

    def set_length(self, seq: int, n: int):
        self.seqs[seq, 0] = n

    def set_token(self, seq: int, tok: int):
        self.seqs[seq, 1] = tok

    def token(self, seq: int = 0) -> int:
        return int(self.seqs[seq, 1].item())


class SequenceStates(SlotStates):
    """Lengths + caches of all slots of the hybrid decoder."""

    def __init__(self, cfg: QwenConfig, spec: ShardSpec, max_seq_len: int, max_batch: int, device):
        super().__init__(max_batch, device)
        self.kv = KVCache(cfg, spec, max_seq_len, max_batch, device)
        self.dn = DeltaNetState(cfg, spec, max_batch, device)

    def reset(self, seq: Optional[int] = None):
        if seq is None:
            self.seqs.zero_()
            self.dn.S.zero_()
            self.dn.conv.zero_()
        else:
            self.seqs[seq].zero_()
            self.dn.S[:, seq].zero_()
            self.dn.conv[:, seq].zero_()

    def snapshot(self, seq: int = 0, with_kv: bool = False) -> SequenceSnapshot:
        """KV entries beyond the snapshotted length are never visible again after
        a restore, so the cache itself only needs copying for full checkpoints."""
        n = self.length(seq)
        return SequenceSnapshot(
            seq, n, self.token(seq),
            self.kv.k[:, seq, :n].clone() if with_kv else None,
            self.kv.v[:, seq, :n].clone() if with_kv else None,
            self.dn.S[:, seq].clone(), self.dn.conv[:, seq].clone())

    def restore(self, snap: SequenceSnapshot, seq: Optional[int] = None):
        seq = snap.seq if seq is None else seq
        self.seqs[seq, 0] = snap.length
        self.seqs[seq, 1] = snap.token
        self.dn.S[:, seq].copy_(snap.S)
        self.dn.conv[:, seq].copy_(snap.conv)
        if snap.k is not None:
            self.kv.k[:, seq, :snap.length].copy_(snap.k)
            self.kv.v[:, seq, :snap.length].copy_(snap.v)

    def state_dict(self, seq: int = 0) -> Dict[str, torch.Tensor]:
        """Host-serialisable checkpoint of one sequence."""
        s = self.snapshot(seq, with_kv=True)
        return {"length": torch.tensor(s.length), "token": torch.tensor(s.token), "k": s.k.cpu(),
                "v": s.v.cpu(), "S": s.S.cpu(), "conv": s.conv.cpu()}

    def load_state_dict(self, sd: Dict[str, torch.Tensor], seq: int = 0):
        dev = self.seqs.device
        self.restore(SequenceSnapshot(seq, int(sd["length"]), int(sd["token"]), sd["k"].to(dev),
                                      sd["v"].to(dev), sd["S"].to(dev), sd["conv"].to(dev)), seq)


@dataclass
class MixerSnapshot:
    """Device copy of everything position-dependent for one slot of a `MixerStates`."""
    seq: int
    length: int
    token: int
    kv: Optional[List[tuple]]
    state: List[tuple]


class MixerStates(SlotStates):
    """Slots of a decoder whose layers are described one by one.  Every run of a layer
    has arrays of its own (layers may differ in size, and one that shares another's
    weights, or runs several times, still has its own history): K and V rows
    [slot][max_seq][kv_heads][dim padded to 8] in the element type, the recurrent state
    [slot][heads][state][vdim] in fp32, and the convolution's last taps - 1 inputs
    [slot][taps-1][channels].  What a run has not is an array of size zero."""

    def __init__(self, cfg, max_seq_len: int, max_batch: int, device, dtype: torch.dtype):
        super().__init__(max_batch, device)
        self.max_seq_len = max_seq_len
        z = lambda *sh, dt=dtype: torch.zeros(*sh, dtype=dt, device=device)
        self.k, self.v, self.S, self.conv = [], [], [], []
        for a, s in cfg.run_mixers():
            G, dp, vp = (a.kv_heads, -(-a.dim // 8) * 8, -(-a.vd // 8) * 8) if a is not None else (0, 8, 8)
            self.k.append(z(max_batch, max_seq_len, G, dp))
            self.v.append(z(max_batch, max_seq_len, G, vp))
            heads, N, P, taps, ch = (s.heads, s.state, s.vdim, s.conv, s.conv_channels) if s is not None else (0, 1, 1, 1, 0)
            self.S.append(z(max_batch, heads, N, P, dt=torch.float32))
            self.conv.append(z(max_batch, taps - 1, ch))

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for ts in (self.k, self.v, self.S, self.conv) for t in ts)

    def reset(self, seq: Optional[int] = None):
        sl = slice(None) if seq is None else seq
        self.seqs[sl].zero_()
        for t in self.S + self.conv:
            t[sl].zero_()

    def snapshot(self, seq: int = 0, with_kv: bool = False) -> MixerSnapshot:
        n = self.length(seq)
        return MixerSnapshot(seq, n, self.token(seq),
                             [(k[seq, :n].clone(), v[seq, :n].clone()) for k, v in zip(self.k, self.v)] if with_kv else None,
                             [(S[seq].clone(), c[seq].clone()) for S, c in zip(self.S, self.conv)])

    def restore(self, snap: MixerSnapshot, seq: Optional[int] = None):
        seq = snap.seq if seq is None else seq
        self.seqs[seq, 0], self.seqs[seq, 1] = snap.length, snap.token
        for (S, c), tS, tc in zip(snap.state, self.S, self.conv):
            tS[seq].copy_(S)
            tc[seq].copy_(c)
        for (k, v), tk, tv in zip(snap.kv or [], self.k, self.v):
            tk[seq, :snap.length].copy_(k)
            tv[seq, :snap.length].copy_(v)

    def state_dict(self, seq: int = 0) -> Dict[str, torch.Tensor]:
        """Host-serialisable checkpoint of one sequence."""
        s = self.snapshot(seq, with_kv=True)
        out = {"length": torch.tensor(s.length), "token": torch.tensor(s.token)}
        for i, ((k, v), (S, c)) in enumerate(zip(s.kv, s.state)):
            out.update({f"k{i}": k.cpu(), f"v{i}": v.cpu(), f"S{i}": S.cpu(), f"conv{i}": c.cpu()})
        return out

    def load_state_dict(self, sd: Dict[str, torch.Tensor], seq: int = 0):
        n = range(len(self.S))
        self.restore(MixerSnapshot(seq, int(sd["length"]), int(sd["token"]), [(sd[f"k{i}"], sd[f"v{i}"]) for i in n],
                                   [(sd[f"S{i}"], sd[f"conv{i}"]) for i in n]), seq)
