"""A plain, slow implementation of the Degedra decoder for the tests: one function per mechanism,
written from the equations, sharing nothing with the product code.  Everything runs in the dtype of
the tensors it is given (the tests use float64 or float32 on the CPU).

Notation: t, s are token indices of one sequence; matrices are stored [out, in] and applied as W x.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def linear(W, x):
    return x @ W.to(x.dtype).T


def rotate_half(x, pos, dims, base):
    """x [tokens, heads, dim]; the first `dims` of every head turn in the pairs (i, i + dims/2)."""
    h = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(h)], dtype=torch.float64)
    a = pos.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :h], x[..., h:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def window_attention(q, k, v, scale, window, q0=0):
    """q [n, H, d] at positions q0 .. q0+n-1; k [m, G, d], v [m, G, e] at positions 0 .. m-1."""
    n, H, _ = q.shape
    m, G, _ = k.shape
    out = torch.zeros(n, H, v.shape[-1], dtype=q.dtype)
    for i in range(n):
        p = q0 + i
        lo = max(0, p - window + 1)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:p + 1, g] @ q[i, h]) * scale
            w = torch.exp(s - s.max())
            out[i, h] = (w / w.sum()) @ v[lo:p + 1, g]
    return out


def attention_branch(c, eps, W, p, x, pos0, cache):
    """Left branch.  `cache`: dict with 'k', 'v' of earlier tokens (or empty); extended in place."""
    H, G, d = c["heads"], c["kv_heads"], c["dim"]
    n = x.shape[0]
    pos = torch.arange(pos0, pos0 + n)
    q, k = linear(W[p + "q"], x), linear(W[p + "k"], x)
    v = k.reshape(n, G, d)
    q = (rms(q, eps) * W[p + "q.norm"].to(x.dtype)).reshape(n, H, d)
    k = (rms(k, eps) * W[p + "k.norm"].to(x.dtype)).reshape(n, G, d)
    q = rotate_half(q, pos, c["rot"]["dims"], c["rot"]["base"])
    k = rotate_half(k, pos, c["rot"]["dims"], c["rot"]["base"])
    cache["k"] = torch.cat([cache["k"], k]) if "k" in cache else k
    cache["v"] = torch.cat([cache["v"], v]) if "v" in cache else v
    o = window_attention(q, cache["k"], cache["v"], c["scale"], c["mask"]["size"], pos0)
    return linear(W[p + "o"], o.reshape(n, H * d))


def causal_conv_silu(u, W, b, hist):
    """u [n, channels], hist [taps-1, channels] (zeros before the start) -> (silu(conv), new hist)."""
    taps = W.shape[1]
    full = torch.cat([hist, u])
    y = torch.stack([sum(W[:, j].to(u.dtype) * full[t + j] for j in range(taps)) + b.to(u.dtype)
                     for t in range(u.shape[0])])
    return silu(y), full[full.shape[0] - (taps - 1):]


def ssd_recurrence(x, B, C, dt, A_log, D, S):
    """x [n, heads, P], B, C [n, groups, N], dt [n, heads] (already positive); S [heads, N, P] is
    the state before the first token.  Returns (y [n, heads, P], state after the last token)."""
    n, H, P = x.shape
    rep = H // B.shape[1]
    y = torch.zeros_like(x)
    S = S.clone()
    for t in range(n):
        for h in range(H):
            g = h // rep
            a = torch.exp(-torch.exp(A_log[h].to(x.dtype)) * dt[t, h])
            S[h] = a * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h].to(x.dtype) * x[t, h]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    u = y * silu(z)
    n, I = u.shape
    return rms(u.reshape(n, groups, I // groups), eps).reshape(n, I) * w.to(y.dtype)


def ssd_branch(c, eps, W, p, x, state):
    """Right branch.  `state`: dict with 'S' and 'conv' (or empty: zeros); replaced in place."""
    H, P, N, Gr = c["heads"], c["vdim"], c["state"], c["groups"]
    I, n = H * P, x.shape[0]
    u = linear(W[p + "in"], x)
    z, xbc, dt = u[:, :I], u[:, I:2 * I + 2 * Gr * N], u[:, 2 * I + 2 * Gr * N:]
    if "S" not in state:
        state["S"] = torch.zeros(H, N, P, dtype=x.dtype)
        state["conv"] = torch.zeros(W[p + "conv"].shape[1] - 1, I + 2 * Gr * N, dtype=x.dtype)
    xbc, state["conv"] = causal_conv_silu(xbc, W[p + "conv"], W[p + "conv.b"], state["conv"])
    dt = softplus(dt + W[p + "dt_bias"].to(x.dtype))
    y, state["S"] = ssd_recurrence(xbc[:, :I].reshape(n, H, P), xbc[:, I:I + Gr * N].reshape(n, Gr, N),
                                   xbc[:, I + Gr * N:].reshape(n, Gr, N), dt, W[p + "A_log"], W[p + "D"],
                                   state["S"])
    y = gated_group_norm(y.reshape(n, I), u[:, :I], W[p + "norm"], c["norm_groups"], eps)
    return linear(W[p + "o"], y)


def mlp(W, p, x):
    return linear(W[p + "down"], silu(linear(W[p + "gate"], x)) * linear(W[p + "up"], x))


class Oracle:
    """One sequence at a time; `cfg` is the parsed config.json, `W` name -> tensor."""

    def __init__(self, cfg, W, dtype=torch.float64):
        self.cfg, self.dtype = cfg, dtype
        self.W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in W.items()}
        self.reset()

    def reset(self):
        self.pos = 0
        self.caches = [{} for _ in self.cfg["layers"]]
        self.states = [{} for _ in self.cfg["layers"]]

    def forward(self, tokens, layers_out=None):
        """Feed tokens; returns logits [n, vocab].  `layers_out`: list that receives the residual
        stream after every layer."""
        W, cfg = self.W, self.cfg
        eps = cfg["norm"]["eps"]
        x = W["embed"][torch.as_tensor(tokens)].clone()
        for i, L in enumerate(cfg["layers"]):
            src = i
            while cfg["layers"][src].get("weights_of") is not None:
                src = cfg["layers"][src]["weights_of"]
            p, m = f"l{src}.", L["mixer"]
            left = attention_branch(m["left"], eps, W, p + "mix.left.", x, self.pos, self.caches[i])
            right = ssd_branch(m["right"], eps, W, p + "mix.right.", x, self.states[i])
            mixed = m["left_scale"] * left + m["right_scale"] * right
            x = x + rms(mixed, eps) * W[p + "norm1"]
            if L.get("mlp") is not None:
                x = x + rms(mlp(W, p + "mlp.", x), eps) * W[p + "norm2"]
            if layers_out is not None:
                layers_out.append(x.clone())
        self.pos += len(tokens)
        lg = linear(W["head"], rms(x, eps) * W["final.norm"])
        cap = cfg.get("logit_softcap")
        return cap * torch.tanh(lg / cap) if cap else lg

    def greedy(self, prompt, n_new):
        self.reset()
        out = [int(self.forward(prompt)[-1].argmax())]
        while len(out) < n_new:
            out.append(int(self.forward(out[-1:])[-1].argmax()))
        return out
