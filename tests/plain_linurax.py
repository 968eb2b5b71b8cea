"""Linurax, written out plainly: one function per mechanism on whole sequences, slow, in float64 (or whatever type the
tensors come in). Shares no code with the package; the engine's tests compare against it.

Notation: W x is a matrix stored [out, in] applied to a column; t, i, j count positions from 0 in a sequence.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def turn_neighbours(x, positions, base: float, dims: int):
    """x [T, heads, d]: numbers (2 n, 2 n + 1) of every head's first ``dims`` are turned by position * base^(-2 n / dims)."""
    n = torch.arange(dims // 2, dtype=torch.float64)
    angle = positions.to(torch.float64)[:, None] * (float(base) ** (-2.0 * n / dims))[None, :]
    c, s = torch.cos(angle).to(x.dtype)[:, None, :], torch.sin(angle).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def talking_scores(q, k, scale: float, talk):
    """q [T, H, d], k [T, G, d] -> [H, T, T]: scaled dot products of every query head with its key head, then every head's
    scores become a weighted sum of all heads' scores (weights ``talk`` [H, H], row = the head that receives)."""
    H, G = q.shape[1], k.shape[1]
    kk = k.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    return torch.einsum("hg,gij->hij", talk, s)


def sigmoid_weights(scores, bias, seen=None):
    """[H, T, T] scores and a number per head -> weights sigmoid(score + bias) of the keys j <= i, zero elsewhere. ``seen``
    [T, T] takes the place of j <= i (a test asks what a lost key would do)."""
    T = scores.shape[-1]
    seen = torch.ones((T, T), dtype=torch.bool).tril() if seen is None else seen
    return torch.where(seen, torch.sigmoid(scores + bias[:, None, None]), torch.zeros((), dtype=scores.dtype))


def attention(h, p: Dict[str, torch.Tensor], pre: str, m: dict, eps: float, seen=None, stored=lambda t: t):
    T = h.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q, k = h @ p[pre + "q"].T, h @ p[pre + "k"].T
    v = stored(k.view(T, G, d))                            # the keys as projected are the values
    q = rms(q, p[pre + "q.norm"], eps).view(T, H, d)       # one root mean square over all heads together
    k = rms(k, p[pre + "k.norm"], eps).view(T, G, d)
    if m.get("rot"):
        pos = torch.arange(T)
        q = turn_neighbours(q, pos, m["rot"]["base"], int(m["rot"]["dims"]))
        k = turn_neighbours(k, pos, m["rot"]["base"], int(m["rot"]["dims"]))
    q, k = stored(q), stored(k)
    w = sigmoid_weights(talking_scores(q, k, float(m["scale"]), p[pre + "talk"]), p[pre + "pb"], seen)
    o = torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(H // G, dim=1)).reshape(T, H * d)
    return (o * torch.sigmoid(h @ p[pre + "g"].T)) @ p[pre + "o"].T


def mingru_states(z, u):
    """z, u [T, C] (the gate and the raw candidate): S_t = (1 - z_t) S_(t-1) + z_t c(u_t), S_-1 = 0, with c(u) = u + 1/2
    from zero on and sigmoid(u) below."""
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        out.append(S)
    return torch.stack(out)


def mingru(h, p: Dict[str, torch.Tensor], pre: str):
    z = torch.sigmoid(h @ p[pre + "z"].T + p[pre + "z.b"])
    u = h @ p[pre + "x"].T + p[pre + "x.b"]
    return (mingru_states(z, u) * silu(h @ p[pre + "g"].T)) @ p[pre + "o"].T


def feed_forward(h, p: Dict[str, torch.Tensor], pre: str):
    return (silu(h @ p[pre + "gate"].T) * (h @ p[pre + "up"].T)) @ p[pre + "down"].T


def forward(cfg: dict, p: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None, dtype=torch.float64,
            round_to=None, seen=None):
    """Logits [T, vocab] of one sequence in ``dtype``; ``layers_out`` collects the stream after every layer. ``round_to``:
    what the sublayers read, and an attention's queries, keys and values, are rounded to this type on the way (what a 16-bit
    engine does at least)."""
    p = {k: v.to(dtype) for k, v in p.items()}
    eps = float(cfg["norm"]["eps"])

    def read(x):
        return x.to(round_to).to(dtype) if round_to is not None else x

    x = p["embed"][torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        if layer["type"] == "attention":
            a = attention(read(x), p, pre + "mix.", layer["mixer"], eps, seen, stored=read)
        elif layer["type"] == "mingru":
            a = mingru(read(x), p, pre + "mix.")
        else:
            raise ValueError(layer["type"])
        x = x + rms(a, p[pre + "norm1"], eps)              # the norm sits on the sublayer's output
        if layer.get("mlp"):
            x = x + rms(feed_forward(read(x), p, pre + "mlp."), p[pre + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return read(rms(x, p["final.norm"], eps)) @ p["embed"].T
