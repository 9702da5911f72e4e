"""Plain float64 restatement of the Kazolorn design, one function per mechanism; shares no code with the served model.

Notation: ``P`` maps tensor names to float64 tensors, ``cfg`` is the checkpoint's ``config.json`` as a dict, token rows are
the leading dimension.  Block ``i`` gives ``r_(i+1) = x + ls1 * mixer(n1(x)) + ls2 * ff(n2(x))`` with two RMS norms of the same
``x``; what enters the next block is a weighted sum of ``r_(i+1)`` and everything before it (``r_0`` is the embedding row).
"""
from __future__ import annotations

import math
from typing import Dict, List, Tuple

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ------------------------------------------------------------------------------------------------ attention
def in_window(T: int, window: int) -> torch.Tensor:
    """[query, key] booleans: the query itself and the ``window - 1`` tokens before it (0: all earlier ones)"""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < window) if window > 0 else d >= 0


def head_slopes(H: int) -> List[float]:
    return [2.0 ** (-8.0 * (n + 1) / H) for n in range(H)]


def biased_scores(q: torch.Tensor, k: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, D], k [T, G, D] -> [H, T, T]: scaled products minus the head's slope times the distance"""
    T, H, _ = q.shape
    G = k.shape[1]
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(F64)
    return torch.stack([(q[:, n] @ k[:, n // (H // G)].T) * scale - s * dist for n, s in enumerate(head_slopes(H))])


def mix_heads(scores: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """row n of the result is the ``talk[n]``-weighted sum of all heads' scores"""
    out = torch.zeros_like(scores)
    for n in range(talk.shape[0]):
        for g in range(talk.shape[1]):
            out[n] += talk[n, g] * scores[g]
    return out


def softmax_plus_one(s: torch.Tensor, ok: torch.Tensor) -> torch.Tensor:
    """exp(s) / (1 + sum of exp(s)) over the visible keys"""
    s = s.masked_fill(~ok, -float("inf"))
    top = s.max(-1, keepdim=True).values.clamp_min(0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention(h: torch.Tensor, P: Dict, p: str, m: Dict) -> torch.Tensor:
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ P[p + "q"].T + P[p + "q.b"]).view(T, H, D)
    k = (h @ P[p + "k"].T + P[p + "k.b"]).view(T, G, D)
    s = mix_heads(biased_scores(q, k, m["scale"]), P[p + "talk"])
    ok = in_window(T, int((m.get("mask") or {}).get("size", 0)))
    rows = [softmax_plus_one(s[n], ok) @ k[:, n // (H // G)] for n in range(H)]         # the keys are the values
    return torch.cat(rows, -1) @ P[p + "o"].T + P[p + "o.b"]


# ------------------------------------------------------------------------------------------------ feed-forward
def poly_norm(z: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return w[0] * rms(z, eps) + w[1] * rms(z ** 2, eps) + w[2] * rms(z ** 3, eps) + w[3]


def dense_ff(h: torch.Tensor, P: Dict, p: str, eps: float) -> torch.Tensor:
    return poly_norm(h @ P[p + "up"].T, P[p + "act"], eps) @ P[p + "down"].T


def gated_expert(h: torch.Tensor, P: Dict, p: str) -> torch.Tensor:
    g = h @ P[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def choose(z: torch.Tensor, top: int) -> Tuple[List[List[int]], List[List[float]]]:
    """per token: the ``top`` experts of largest sigmoid score (lowest index among equals) with the scores as they are"""
    idx, wts = [], []
    for row in z.tolist():
        order = sorted(range(len(row)), key=lambda j: (-row[j], j))[:top]
        idx.append(order)
        wts.append([1.0 / (1.0 + math.exp(-row[j])) for j in order])
    return idx, wts


def routed_ff(h: torch.Tensor, P: Dict, p: str, top: int) -> torch.Tensor:
    """the score scales what goes INTO the expert"""
    idx, wts = choose(h @ P[p + "router"].T, top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j, w in zip(idx[t], wts[t]):
            out[t] += gated_expert(w * h[t:t + 1], P, f"{p}e{j}.")[0]
    return out


# ------------------------------------------------------------------------------------------------ the model
def depth_average(rows: List[torch.Tensor], w: torch.Tensor) -> torch.Tensor:
    x = torch.zeros_like(rows[0])
    for j, r in enumerate(rows):
        x = x + w[j] * r
    return x


def forward(cfg: Dict, P: Dict, tokens: List[int]):
    """-> (logits [T, vocab], what leaves every layer: the depth averages)"""
    P = {k: v.to(F64) for k, v in P.items()}
    eps = cfg["norm"]["eps"]
    x = P["embed"][torch.tensor(tokens)]
    rows, trail = [x], []
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = P[p + "ls1"] * attention(rms(x, eps) * P[p + "norm1"], P, p + "mix.", lay["mixer"])
        mlp = lay.get("mlp")
        if mlp:
            h = rms(x, eps) * P[p + "norm2"]
            f = dense_ff(h, P, p + "mlp.", eps) if mlp["kind"] == "dense" else routed_ff(h, P, p + "mlp.", mlp["router"]["top"])
            y = y + P[p + "ls2"] * f
        rows.append(x + y)
        x = depth_average(rows, P[p + "dwa"])
        trail.append(x)
    return (rms(x, eps) * P["final.norm"]) @ P["head"].T, trail
