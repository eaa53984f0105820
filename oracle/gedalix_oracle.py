"""Plain restatement of the Gedalix design: one function per mechanism, no cache, no batching, keys and values expanded per head.

Slow on purpose and independent of the engine: it shares no code with the package, takes the config dictionary and the
tensors by their checkpoint names, and computes in one floating type (float64 by default) from the bf16 weight values.
The reference service names models by tag and has no model code (app/utils/config.py:86), so nothing here restates it.

Notation: x the residual stream [T, W]; h what a sublayer reads; c the latent of a token; p its position in the sequence.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * gain over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def turn_halves(x: torch.Tensor, pos: torch.Tensor, base: float) -> torch.Tensor:
    """Coordinates (i, i + d / 2) of the last axis turned by pos * base^(-2 i / d); x is [T, ..., d]."""
    d = x.shape[-1]
    if d == 0:
        return x
    half = d // 2
    f = base ** (-2.0 * torch.arange(half, dtype=x.dtype) / d)
    ang = (pos.to(x.dtype)[:, None] * f).reshape(x.shape[0], *([1] * (x.dim() - 2)), half)
    a, b = x[..., :half], x[..., half:]
    return torch.cat([a * torch.cos(ang) - b * torch.sin(ang), b * torch.cos(ang) + a * torch.sin(ang)], -1)


def attend_with_sink(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, sink: torch.Tensor) -> torch.Tensor:
    """q, k [T, H, D], v [T, H, V] -> [T, H * V]: causal softmax whose denominator holds exp(sink_h) once more, unscaled and
    without a value."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril(), -torch.inf)
    s = torch.cat([s, sink[:, None, None].expand(-1, T, 1)], -1)
    return torch.einsum("hij,jhv->ihv", torch.softmax(s, -1)[..., :T], v).reshape(T, -1)


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    """Latent attention with a rotated key part shared by the heads, a sink per head and an element-wise output gate."""
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = float((m.get("rot") or {}).get("base", 1.0))
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T).reshape(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :C], w[p + "dkv.norm"], eps)
    shared = turn_halves(down[:, C:], pos, base)[:, None].expand(T, H, R)
    q = torch.cat([q[..., :D], turn_halves(q[..., D:], pos, base)], -1)
    k = torch.cat([(c @ w[p + "uk"].T).reshape(T, H, D), shared], -1)
    v = (c @ w[p + "uv"].T).reshape(T, H, V)
    o = attend_with_sink(q, k, v, m["scale"], w[p + "sink"])
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, top: int):
    """Expert numbers [T, top] with the largest biased logits, and the softmax over those logits."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best, ids = torch.topk(z, top, -1)
    return ids, torch.softmax(best, -1)


def expert_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: Dict) -> torch.Tensor:
    """Softmax-weighted chosen experts, plus the shared expert times one sigmoid gate per token."""
    out = torch.zeros_like(h)
    ids, wt = choose(h, w, p, mlp["router"]["top"])
    for t in range(h.shape[0]):
        for e, s in zip(ids[t].tolist(), wt[t]):
            out[t] += s * gated_ff(h[t][None], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * gated_ff(h, w, p + "shared.")
    return out


# ------------------------------------------------------------------------------------------------ the whole
def embedding(tokens: List[int], w: Dict[str, torch.Tensor], scale: float) -> torch.Tensor:
    return w["embed"][torch.tensor(tokens)] * scale + w["pos"][:len(tokens)]


def layer(x: torch.Tensor, w: Dict[str, torch.Tensor], i: int, l: Dict, eps: float, mult: float) -> torch.Tensor:
    p = f"l{i}."
    x = x + mult * w[p + "ls1"] * latent_attention(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", l["mixer"], eps)
    if l.get("mlp"):
        x = x + mult * w[p + "ls2"] * expert_ff(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", l["mlp"])
    return x


def runs(cfg: Dict) -> List[tuple]:
    """(layer, pass or None) in the order they run; the pass number stands only at a pass's first layer."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + body + [(i, None) for i in range(b, n)]


def forward(cfg: Dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            trail: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab]; `trail` collects the stream after every layer run."""
    w = {k: v.to("cpu", dtype) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    first = embedding(tokens, w, float(cfg["embedding"]["scale"]))
    x = first
    for i, t in runs(cfg):
        if t is not None:                      # what comes right before a pass of the loop
            x = (x + first if t > 0 else x) + w["loop.step"][t]
        x = layer(x, w, i, cfg["layers"][i], eps, float(cfg["residual_mult"]))
        if trail is not None:
            trail.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
