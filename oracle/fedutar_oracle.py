"""Plain restatement of the Fedutar design: one function per mechanism, no cache, no batching, the recurrence token by token.

Slow on purpose and independent of the engine: it shares no code with the package, takes the config dictionary and the
tensors by their checkpoint names, and computes in one floating type (float64 by default) from the bf16 weight values.
The reference service names models by tag and has no model code (app/utils/config.py:86), so nothing here restates it.

Notation: x the residual stream [T, W]; h what a sublayer reads; S a matrix state [key dim, value dim] per head; p a position.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * gain over the last axis."""
    return unit_rms(x, eps) * gain


# ------------------------------------------------------------------------------------------------ softmax attention
def temperature(T: int, coef: float, every: int, dtype) -> torch.Tensor:
    """Factor of the query at every position: 1 + coef ln(1 + floor((p + 1) / every))."""
    return torch.tensor([1.0 + coef * math.log(1 + (p + 1) // every) for p in range(T)], dtype=dtype)


def causal_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H * V]; query head h reads key head h // (H / G)."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    hidden = ~torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(hidden, -torch.inf)
        out[:, h] = torch.softmax(s, -1) @ v[:, g]
    return out.reshape(T, -1)


def softmax_side(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    """Grouped-query attention without positions: normed queries and keys, a temperature that grows with the position, and an
    element-wise gate on the heads."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[p + "q"].T).reshape(T, H, D), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].T).reshape(T, G, D), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).reshape(T, G, V)
    if m.get("q_temp"):
        q = q * temperature(T, m["q_temp"]["coef"], int(m["q_temp"]["every"]), h.dtype)[:, None, None]
    o = causal_attention(q, k, v, m["scale"])
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ retention
def turn_halves(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """Coordinates (i, i + dims / 2), i < dims / 2, turned by pos * base^(-2 i / dims); x is [T, heads, D], the rest passes."""
    if dims == 0:
        return x
    half = dims // 2
    f = base ** (-2.0 * torch.arange(half, dtype=x.dtype) / dims)
    ang = (pos.to(x.dtype)[:, None] * f)[:, None]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * torch.cos(ang) - b * torch.sin(ang), b * torch.cos(ang) + a * torch.sin(ang), x[..., dims:]], -1)


def retain(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: List[float]) -> torch.Tensor:
    """S <- decay S + k v^T, o = S^T q, token by token; [T, H, D], [T, H, D], [T, H, V] -> [T, H, V]."""
    T, H, D = q.shape
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    d = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def retention_side(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    pos = torch.arange(T)
    q = turn_halves((h @ w[p + "q"].T).reshape(T, H, D), pos, int(rot["dims"]), float(rot["base"]))
    k = turn_halves((h @ w[p + "k"].T).reshape(T, H, D), pos, int(rot["dims"]), float(rot["base"])) * D ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    o = unit_rms(retain(q, k, v, m["decay"]), eps).reshape(T, H * V)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    return (m["left_scale"] * softmax_side(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * retention_side(h, w, p + "right.", m["right"], eps))


# ------------------------------------------------------------------------------------------------ feed-forward
def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    lin = lambda z, n: z @ w[p + n].T + w[p + n + ".b"]
    return lin(silu(lin(h, "gate")) * lin(h, "up"), "down")


def clipped_expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, top: int):
    """Expert numbers [T, top] with the largest logits, and the softmax over those logits."""
    best, ids = torch.topk(h @ w[p + "router"].T, top, -1)
    return ids, torch.softmax(best, -1)


def expert_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: Dict) -> torch.Tensor:
    out = torch.zeros_like(h)
    ids, wt = choose(h, w, p, mlp["router"]["top"])
    for e in range(mlp["router"]["experts"]):
        rows, place = (ids == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += wt[rows, place][:, None] * clipped_expert(h[rows], w, f"{p}e{e}.", float(mlp["expert"]["limit"]))
    return out


def feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: Dict) -> torch.Tensor:
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else expert_ff(h, w, p, mlp)


# ------------------------------------------------------------------------------------------------ the whole
def layer(x: torch.Tensor, w: Dict[str, torch.Tensor], i: int, l: Dict, eps: float) -> torch.Tensor:
    p = f"l{i}."
    y = parallel_mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", l["mixer"], eps)
    x = x + rms_norm(y, w[p + "norm1b"], eps)
    if l.get("mlp"):
        y = feed_forward(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", l["mlp"])
        x = x + rms_norm(y, w[p + "norm2b"], eps)
    return x


def runs(cfg: Dict) -> List[tuple]:
    """(layer, does a pass of the loop begin here) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body + [(i, False) for i in range(b, n)]


def head(x: torch.Tensor, w: Dict[str, torch.Tensor], cfg: Dict, eps: float) -> torch.Tensor:
    z = rms_norm(x, w["final.norm"], eps) @ w["embed"].T * float(cfg.get("logit_scale", 1.0))
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z


def forward(cfg: Dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            trail: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab]; `trail` collects the stream after every layer run."""
    w = {k: v.to("cpu", dtype) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    first = w["embed"][torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    x = first
    for i, begins in runs(cfg):
        if begins:
            x = torch.cat([x, first], -1) @ w["loop.in"].T
        x = layer(x, w, i, cfg["layers"][i], eps)
        if trail is not None:
            trail.append(x)
    return head(x, w, cfg, eps)
