"""A plain, slow implementation of the Vekerax decoder for the tests: one function per mechanism, written
from the equations, sharing nothing with the product code.  Everything runs in the dtype of the tensors it
is given (float64 on the CPU in the tests).

Notation: i, j are token positions of one sequence; matrices are stored [out, in] and applied as W x.
"""
from __future__ import annotations

import math

import torch

from degedra_oracle import linear, rms, silu


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def relu_mlp(W, p, x):
    """W_down (max(W_gate x, 0) * W_up x)"""
    return linear(W[p + "down"], torch.clamp(linear(W[p + "gate"], x), min=0) * linear(W[p + "up"], x))


def head_norm(x, w, eps):
    """x [tokens, heads, dim]: every head over its own root mean square, times one weight for all heads."""
    return rms(x, eps) * w.to(x.dtype)


def visible(i, j, window, keep):
    """Does the token at position i see the one at j?  window None: all earlier tokens."""
    return j <= i and (window is None or i - j < window or j < keep)


def sink_attention(q, k, v, scale, softcap=None, window=None, keep=0, sink=None, q0=0):
    """q [n, H, d] at positions q0 .. q0+n-1; k [m, G, d], v [m, G, e] at positions 0 .. m-1; sink [H]:
    one more term exp(sink) in the denominator."""
    n, H, _ = q.shape
    m, G, _ = k.shape
    out = torch.zeros(n, H, v.shape[-1], dtype=q.dtype)
    for r in range(n):
        i = q0 + r
        seen = torch.tensor([j for j in range(min(m, i + 1)) if visible(i, j, window, keep)])
        for h in range(H):
            g = h // (H // G)
            s = (k[seen, g] @ q[r, h]) * scale
            if softcap:
                s = softcap * torch.tanh(s / softcap)
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h].to(s.dtype))
            w = torch.exp(s - top)
            den = w.sum() + (0 if sink is None else torch.exp(sink[h].to(s.dtype) - top))
            out[r, h] = (w / den) @ v[seen, g]
    return out


def attention_mixer(c, eps, W, p, x, cache):
    """`cache`: dict with 'k', 'v' of earlier tokens (or empty); extended in place."""
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    n = x.shape[0]
    q = head_norm(linear(W[p + "q"], x).reshape(n, H, d), W[p + "q.norm"], eps)
    k = head_norm(linear(W[p + "k"], x).reshape(n, G, d), W[p + "k.norm"], eps)
    v = linear(W[p + "v"], x).reshape(n, G, e)
    q0 = cache["k"].shape[0] if "k" in cache else 0
    cache["k"] = torch.cat([cache["k"], k]) if q0 else k
    cache["v"] = torch.cat([cache["v"], v]) if q0 else v
    mask = c.get("mask") or {}
    o = sink_attention(q, cache["k"], cache["v"], c["scale"], c.get("softcap"), mask.get("size"), mask.get("keep_first") or 0,
                       W[p + "sink"], q0)
    return linear(W[p + "o"], o.reshape(n, H * e))


def decayed_outer_recurrence(q, k, v, decay, S):
    """Every token fades a head's matrix by the head's constant, adds the outer product of its key and value, and
    reads the result with its query; q, k [n, heads, dim], v [n, heads, vdim], S [heads, dim, vdim].  Returns (o [n, heads, vdim], last state)."""
    n, H, _ = q.shape
    o = torch.zeros_like(v)
    S = S.clone()
    for t in range(n):
        for h in range(H):
            S[h] = decay[h] * S[h] + torch.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def norm_then_gate(o, g, w, eps):
    """Whole row over its root mean square, times a weight, times sigmoid of the gate."""
    return rms(o, eps) * w.to(o.dtype) * sigmoid(g)


def lightning_mixer(c, eps, W, p, x, state):
    """`state`: dict with 'S' (or empty: zeros); replaced in place."""
    H, d, e = c["heads"], c["dim"], c["vdim"]
    n = x.shape[0]
    q = silu(linear(W[p + "q"], x)).reshape(n, H, d)
    k = silu(linear(W[p + "k"], x)).reshape(n, H, d)
    v = silu(linear(W[p + "v"], x)).reshape(n, H, e)
    S = state.get("S", torch.zeros(H, d, e, dtype=x.dtype))
    o, state["S"] = decayed_outer_recurrence(q, k, v, c["decay"], S)
    return linear(W[p + "o"], norm_then_gate(o.reshape(n, H * e), linear(W[p + "g"], x), W[p + "norm"], eps))


def streams_in(xs, a):
    """xs [streams, n, width] -> their sum weighted by a"""
    return (a.to(xs.dtype)[:, None, None] * xs).sum(0)


def streams_out(xs, M, b, m, y):
    """New streams: column t of M weighs the old ones, plus y times m b[t]."""
    new = torch.zeros_like(xs)
    for t in range(xs.shape[0]):
        for s in range(xs.shape[0]):
            new[t] += M[s, t].to(xs.dtype) * xs[s]
        new[t] += m * b[t].to(xs.dtype) * y
    return new


def layer_order(cfg):
    """Indices of the layers in the order in which they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


class Oracle:
    """One sequence at a time; `cfg` is the parsed config.json, `W` name -> tensor."""

    def __init__(self, cfg, W, dtype=torch.float64):
        self.cfg, self.dtype = cfg, dtype
        self.W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in W.items()}
        self.order = layer_order(cfg)
        self.reset()

    def reset(self):
        self.memory = [{} for _ in self.order]       # cache or state of every run of a layer

    def forward(self, tokens, layers_out=None):
        """Feed tokens; returns logits [n, vocab].  `layers_out`: list that receives the sum of the streams
        after every run of a layer."""
        W, cfg = self.W, self.cfg
        eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
        x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
        hyper = cfg.get("streams")
        xs = torch.stack([x] * (hyper or 1))
        for run, i in enumerate(self.order):
            L, p = cfg["layers"][i], f"l{i}."
            subs = [(1, lambda h: {"attention": attention_mixer, "lightning": lightning_mixer}[L["type"]](
                L["mixer"], eps, W, p + "mix.", h, self.memory[run]))]
            if L.get("mlp") is not None:
                subs.append((2, lambda h: relu_mlp(W, p + "mlp.", h)))
            for q, f in subs:
                hc = f"{p}hc{q}."
                u = streams_in(xs, W[hc + "in"]) if hyper else xs[0]
                y = f(rms(u, eps) * W[f"{p}norm{q}"])
                xs = streams_out(xs, W[hc + "mix"], W[hc + "out"], m, y) if hyper else xs + m * y
            if layers_out is not None:
                layers_out.append(xs.sum(0))
        return linear(W["embed"], rms(xs.sum(0), eps) * W["final.norm"])

    def greedy(self, prompt, n_new):
        self.reset()
        out = [int(self.forward(prompt)[-1].argmax())]
        while len(out) < n_new:
            out.append(int(self.forward(out[-1:])[-1].argmax()))
        return out
