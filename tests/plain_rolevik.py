"""Rolevik, written out plainly: one function per mechanism on whole sequences, slow, in float64 (or whatever type the
tensors come in). Shares no code with the package; the engine's tests compare against it.

Notation: W x is a matrix stored [out, in] applied to a column; t, i, j count positions from 0 in a sequence.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def layer_norm(x, w, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def turn_halves(x, positions, base: float, dims: int):
    """x [T, heads, d]: numbers (n, n + dims / 2) of every head's first ``dims`` are turned by position * base^(-2 n / dims)."""
    half = dims // 2
    n = torch.arange(half, dtype=torch.float64)
    angle = positions.to(torch.float64)[:, None] * (float(base) ** (-2.0 * n / dims))[None, :]
    c, s = torch.cos(angle).to(x.dtype)[:, None, :], torch.sin(angle).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def chunk_mask(T: int, size: Optional[int]):
    """[T, T]: query i sees key j <= i of its own chunk of ``size`` positions (None: every key j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i // size == j // size)


def softmax_attention(q, k, v, scale: float, seen):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv]."""
    H, G = q.shape[1], k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, dim=1)) * scale
    w = torch.softmax(torch.where(seen, s, torch.full((), -math.inf, dtype=s.dtype)), dim=-1)
    return torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(H // G, dim=1)).reshape(q.shape[0], -1)


def attention(h, p: Dict[str, torch.Tensor], pre: str, m: dict, eps: float, seen=None, stored=lambda t: t):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (h @ p[pre + n].T + p[pre + n + ".b"] for n in ("q", "k", "v"))
    q = rms(q, p[pre + "q.norm"], eps).view(T, H, d)       # one root mean square over all heads together
    k = rms(k, p[pre + "k.norm"], eps).view(T, G, d)
    if m.get("rot"):
        pos = torch.arange(T)
        q = turn_halves(q, pos, m["rot"]["base"], int(m["rot"]["dims"]))
        k = turn_halves(k, pos, m["rot"]["base"], int(m["rot"]["dims"]))
    if seen is None:
        seen = chunk_mask(T, int(m["mask"]["size"]) if m.get("mask") else None)
    o = softmax_attention(stored(q), stored(k), stored(v.view(T, G, dv)), float(m["scale"]), seen)
    return o @ p[pre + "o"].T


def causal_filter(x, w, b=None):
    """x [T, C], w [C, taps]: the last column belongs to the current row; rows before the first are zero."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros((taps - 1, x.shape[1]), dtype=x.dtype), x])
    y = sum(padded[j: j + T] * w[:, j] for j in range(taps))
    return y if b is None else y + b


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g, S=None):
    """q, k [T, H, d], v [T, H, dv], beta, g [T, H] -> read-outs [T, H, dv]: the state decays, is corrected towards v along
    k, and is read behind the correction."""
    T, H, d = q.shape
    S = torch.zeros((H, d, v.shape[-1]), dtype=q.dtype) if S is None else S
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def gated_delta(h, p: Dict[str, torch.Tensor], pre: str, m: dict, eps: float):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (silu(causal_filter(h @ p[pre + n].T, p[pre + n + ".conv"])) for n in ("q", "k", "v"))
    q = (unit(q.view(T, G, d)) * d ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(k.view(T, G, d)).repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ p[pre + "b"].T)
    g = torch.exp(-torch.exp(p[pre + "A_log"]) * softplus(h @ p[pre + "a"].T + p[pre + "dt_bias"]))
    o = delta_rule(q, k, v.view(T, H, dv), beta, g)
    o = rms(o, p[pre + "norm"], eps).reshape(T, H * dv) * silu(h @ p[pre + "g"].T)
    return o @ p[pre + "o"].T


def parallel(h, p: Dict[str, torch.Tensor], pre: str, m: dict, eps: float, seen=None, stored=lambda t: t):
    left = attention(h, p, pre + "left.", m["left"], eps, seen, stored)
    right = gated_delta(h, p, pre + "right.", m["right"], eps)
    return 0.5 * (rms(left, p[pre + "left.out"], eps) + rms(right, p[pre + "right.out"], eps))


def block_gates(u, w, b):
    """u [T, C] in equal parts, one matrix [out, in] and one bias a part: sigmoid(w[n] u_n + b[n]), [T, C]."""
    T, n = u.shape[0], w.shape[0]
    return torch.sigmoid(torch.einsum("tni,noi->tno", u.view(T, n, -1), w) + b).reshape(T, -1)


def rglru_states(u, r, i, lam, S=None):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with a = exp(-8 r softplus(lam))."""
    log_a = -8.0 * r * softplus(lam)
    a = torch.exp(log_a)
    put = torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S, out = torch.zeros_like(u[0]) if S is None else S, []
    for t in range(u.shape[0]):
        S = a[t] * S + put[t]
        out.append(S)
    return torch.stack(out)


def rglru(h, p: Dict[str, torch.Tensor], pre: str):
    y = gelu_tanh(h @ p[pre + "y"].T + p[pre + "y.b"])
    u = causal_filter(h @ p[pre + "x"].T + p[pre + "x.b"], p[pre + "conv"], p[pre + "conv.b"])
    r, i = block_gates(u, p[pre + "ra"], p[pre + "ra.b"]), block_gates(u, p[pre + "ri"], p[pre + "ri.b"])
    return (rglru_states(u, r, i, p[pre + "lam"]) * y) @ p[pre + "o"].T


def gated_ff(h, p: Dict[str, torch.Tensor], pre: str, act):
    return (act(h @ p[pre + "gate"].T) * (h @ p[pre + "up"].T)) @ p[pre + "down"].T


def choose(z, correction, top: int, groups: int, keep: int):
    """Router logits [T, n] -> (scores [T, n], chosen [T, top]): scores by softmax; the choice goes by score + correction
    among the members of the ``keep`` groups whose best choice score is largest."""
    s = torch.softmax(z, dim=-1)
    c = s + correction
    T, n = c.shape
    best = c.view(T, groups, n // groups).max(dim=-1).values
    kept = torch.zeros((T, groups), dtype=torch.bool)
    kept.scatter_(1, torch.topk(best, keep, dim=-1).indices, True)
    c = torch.where(kept.repeat_interleave(n // groups, dim=1), c, torch.full((), -math.inf, dtype=c.dtype))
    return s, torch.topk(c, top, dim=-1).indices


def choice_margin(z, correction, top: int, groups: int, keep: int):
    """[T]: how far every row's choice is from another one, in score units: the smaller of the gap between the last kept group
    and the first one left out, and of the gap between the last chosen member and the best one left out."""
    s, chosen = choose(z, correction, top, groups, keep)
    c = s + correction
    T, n = c.shape
    best = c.view(T, groups, n // groups).max(dim=-1).values
    margin = torch.full((T,), math.inf, dtype=c.dtype)
    order = torch.sort(best, dim=-1, descending=True).values
    if keep < groups:
        margin = torch.minimum(margin, order[:, keep - 1] - order[:, keep])
    kept = torch.zeros((T, groups), dtype=torch.bool)
    kept.scatter_(1, torch.topk(best, keep, dim=-1).indices, True)
    open_c = torch.where(kept.repeat_interleave(n // groups, dim=1), c, torch.full((), -math.inf, dtype=c.dtype))
    ranked = torch.sort(open_c, dim=-1, descending=True).values
    if top < (n // groups) * keep:
        margin = torch.minimum(margin, ranked[:, top - 1] - ranked[:, top])
    return margin


def experts(h, p: Dict[str, torch.Tensor], pre: str, m: dict, margins: Optional[list] = None):
    r = m["router"]
    n, identity, top = int(r["experts"]), int(r.get("identity") or 0), int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ p[pre + "router"].T
    s, chosen = choose(z, p[pre + "correction"], top, int(groups["count"]), int(groups["keep"]))
    if margins is not None:
        margins.append(choice_margin(z, p[pre + "correction"], top, int(groups["count"]), int(groups["keep"])))
    scale = 1.0 if r.get("scale") is None else float(r["scale"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen[t].tolist():
            y = h[t] if e >= n else gated_ff(h[t], p, f"{pre}e{e}.", silu)      # behind the experts: the input itself
            out[t] += s[t, e] * scale * y
    if m.get("shared"):
        out = out + gated_ff(h, p, pre + "shared.", silu)
    assert n + identity == s.shape[1]
    return out


def forward(cfg: dict, p: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None, dtype=torch.float64,
            round_to=None, round_scale: float = 1.0, seen=None, margins: Optional[list] = None):
    """Logits [T, vocab] of one sequence in ``dtype``; ``layers_out`` collects the stream after every layer. ``round_to``:
    what the sublayers read, and an attention's queries, keys and values, are rounded to this type on the way (what a 16-bit
    engine does at least), on a grid that ``round_scale`` stretches. ``seen``: a mask in the place of every attention's own (a test asks what a lost key would do);
    ``margins`` collects how near every row's choice of experts was to another one."""
    p = {k: v.to(dtype) for k, v in p.items()}
    eps = float(cfg["norm"]["eps"])

    def read(x):
        return (x * round_scale).to(round_to).to(dtype) / round_scale if round_to is not None else x

    x = p["embed"][torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        if layer["type"] == "parallel":
            a = parallel(read(x), p, pre + "mix.", layer["mixer"], eps, seen, stored=read)
        elif layer["type"] == "rglru":
            a = rglru(read(x), p, pre + "mix.")
        else:
            raise ValueError(layer["type"])
        x = x + layer_norm(a, p[pre + "norm1"], eps) * p[pre + "ls1"]      # norm and scale sit on the sublayer's output
        m = layer.get("mlp")
        if m:
            f = gated_ff(read(x), p, pre + "mlp.", gelu_tanh) if m["kind"] == "dense" else experts(read(x), p, pre + "mlp.", m, margins)
            x = x + layer_norm(f, p[pre + "norm2"], eps) * p[pre + "ls2"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return read(layer_norm(x, p["final.norm"], eps)) @ p["embed"].T * float(cfg.get("logit_scale", 1.0))
