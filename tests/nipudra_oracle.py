"""Plain float64 restatement of the Nipudra design, one function per mechanism; shares no code with the served model.

Notation: ``P`` maps tensor names to float64 tensors, ``cfg`` is the checkpoint's ``config.json`` as a dict, token rows are
the leading dimension.  A layer is ``x += n1b(mixer(n1(x)))``, ``x += n2b(ff(n2(x)))`` (layer norms), then a contribution that
depends on the token itself; recurrences are walked token by token.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ norms, activations
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return rms(d, eps) * w + b


def group_rms(x: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    T, n = x.shape
    return rms(x.view(T, parts, n // parts), eps).reshape(T, n)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def relu_sq(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0.0) ** 2


# ------------------------------------------------------------------------------------------------ positions
def frequencies(rot: Dict) -> Tuple[List[float], float]:
    """(angle per position of every pair, amplitude of cos and sin)"""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def turn(t):
        return n * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turn(s["fast"])), 0), min(math.ceil(turn(s["slow"])), n - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / s["factor"] * r + v * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x: torch.Tensor, rot: Optional[Dict]) -> torch.Tensor:
    """x [T, heads, dim]: channel i of the first ``dims`` turns with channel i + dims / 2"""
    if not rot or not rot["dims"]:
        return x
    f, amp = frequencies(rot)
    h = rot["dims"] // 2
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(f, dtype=F64)[None, :]
    c, s = (torch.cos(a) * amp)[:, None, :], (torch.sin(a) * amp)[:, None, :]
    u, v = x[..., :h], x[..., h:2 * h]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * h:]], -1)


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, channels], w [channels, taps]; the last tap meets the current token"""
    T, C = u.shape
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            k = t - (taps - 1) + j
            if k >= 0:
                y[t] += w[:, j] * u[k]
    return y


# ------------------------------------------------------------------------------------------------ differential attention
def in_window(T: int, window: int) -> torch.Tensor:
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < window) if window > 0 else d >= 0


def keys_values(h: torch.Tensor, P: Dict, p: str, m: Dict):
    """(keys [T, G, 2, dim] after convolution and rotation, values [T, G, vdim] after convolution)"""
    T, G = h.shape[0], m["kv_heads"]
    k = causal_conv(h @ P[p + "k"].T + P[p + "k.b"], P[p + "k.conv"])
    v = causal_conv(h @ P[p + "v"].T + P[p + "v.b"], P[p + "v.conv"])
    k = rotate(k.view(T, G * 2, m["dim"]), m.get("rot")).view(T, G, 2, m["dim"])
    return k, v.view(T, G, m["vdim"])


def diff_lambda(P: Dict, p: str, diff: float) -> float:
    return float(torch.exp((P[p + "lq1"] * P[p + "lk1"]).sum()) - torch.exp((P[p + "lq2"] * P[p + "lk2"]).sum())) + diff


def diff_attention(h: torch.Tensor, P: Dict, p: str, m: Dict, kv, eps: float) -> torch.Tensor:
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    k, v = kv
    q = causal_conv(h @ P[p + "q"].T + P[p + "q.b"], P[p + "q.conv"])
    q = rotate(q.view(T, H * 2, D), m.get("rot")).view(T, H, 2, D)
    ok = in_window(T, int((m.get("mask") or {}).get("size", 0)))
    lam = diff_lambda(P, p, m["diff"])
    heads = []
    for n in range(H):
        g = n // (H // G)
        maps = []
        for a in range(2):
            s = (q[:, n, a] @ k[:, g, a].T) * m["scale"]
            maps.append(torch.softmax(s.masked_fill(~ok, -float("inf")), -1) @ v[:, g])
        heads.append(rms(maps[0] - lam * maps[1], eps) * (1.0 - m["diff"]))
    return torch.cat(heads, -1) @ P[p + "o"].T + P[p + "o.b"]


# ------------------------------------------------------------------------------------------------ recurrences
def ssd_walk(x, B, C, dt, rate, skip) -> torch.Tensor:
    """one head: S <- exp(-rate dt) S + dt B x^T, y = S^T C + skip x;  x [T, V], B and C [T, N], dt [T]"""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=F64)
    out = []
    for t in range(x.shape[0]):
        S = torch.exp(-rate * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        out.append(S.T @ C[t] + skip * x[t])
    return torch.stack(out)


def mamba2(h: torch.Tensor, P: Dict, p: str, m: Dict, eps: float) -> torch.Tensor:
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = torch.split(h @ P[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = silu(causal_conv(xbc, P[p + "conv"]) + P[p + "conv.b"])
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    dt = torch.log1p(torch.exp(-(dt + P[p + "dt_bias"]).abs())) + torch.clamp(dt + P[p + "dt_bias"], min=0.0)
    B, C = B.view(T, G, N), C.view(T, G, N)
    ys = []
    for n in range(H):
        g = n // (H // G)
        ys.append(ssd_walk(x[:, n * V:(n + 1) * V], B[:, g], C[:, g], dt[:, n], torch.exp(P[p + "A_log"][n]), P[p + "D"][n]))
    y = torch.cat(ys, -1) * silu(z)
    return (group_rms(y, m["norm_groups"], eps) * P[p + "norm"]) @ P[p + "o"].T


def decayed_walk(q, k, v, decay: float) -> torch.Tensor:
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    out = []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def retention(h: torch.Tensor, P: Dict, p: str, m: Dict, eps: float) -> torch.Tensor:
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ P[p + "q"].T).view(T, H, D), m.get("rot"))
    k = rotate((h @ P[p + "k"].T).view(T, H, D), m.get("rot")) * D ** -0.5
    v = (h @ P[p + "v"].T).view(T, H, V)
    o = torch.cat([rms(decayed_walk(q[:, n], k[:, n], v[:, n], m["decay"][n]), eps) for n in range(H)], -1)
    return (o * silu(h @ P[p + "g"].T)) @ P[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def expert(h: torch.Tensor, P: Dict, p: str) -> torch.Tensor:
    return relu_sq(h @ P[p + "up"].T) @ P[p + "down"].T


def choose(z: torch.Tensor, top: int):
    """per token: the ``top`` largest logits (lowest index among equals) and the softmax over them alone"""
    idx, wts = [], []
    for row in z.tolist():
        order = sorted(range(len(row)), key=lambda j: (-row[j], j))[:top]
        e = [math.exp(row[j] - row[order[0]]) for j in order]
        idx.append(order)
        wts.append([v / sum(e) for v in e])
    return idx, wts


def routed_ff(h: torch.Tensor, P: Dict, p: str, mlp: Dict) -> torch.Tensor:
    idx, wts = choose(h @ P[p + "router"].T + P[p + "router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j, w in zip(idx[t], wts[t]):
            out[t] += w * expert(h[t:t + 1], P, f"{p}e{j}.")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ P[p + "shared.sg"].T) * expert(h, P, p + "shared.")
    return out


# ------------------------------------------------------------------------------------------------ the model
def token_side(x: torch.Tensor, tokens: torch.Tensor, P: Dict, p: str, layer: int, dim: int, eps: float) -> torch.Tensor:
    e = P["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    g = gelu_tanh(x @ P[p + "side.gate"].T) * e
    return rms(g @ P[p + "side.proj"].T, eps) * P[p + "side.norm"]


def forward(cfg: Dict, P: Dict, tokens: List[int]):
    """-> (logits [T, vocab], the residual after every layer)"""
    P = {k: v.to(F64) for k, v in P.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.tensor(tokens)
    x = P["embed"][ids] * (cfg.get("embedding") or {}).get("scale", 1.0)
    trail, kvs = [], {}
    for i, lay in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", lay["mixer"], lay.get("mlp")

        def norm(v, n):
            return layer_norm(v, P[p + n], P[p + n + ".b"], eps)

        h = norm(x, "norm1")
        if lay["type"] == "attention":
            kvs[i] = kvs[m["kv_from"]] if m.get("kv_from") is not None else keys_values(h, P, p + "mix.", m)
            y = diff_attention(h, P, p + "mix.", m, kvs[i], eps)
        elif lay["type"] == "mamba2":
            y = mamba2(h, P, p + "mix.", m, eps)
        else:
            y = retention(h, P, p + "mix.", m, eps)
        x = x + norm(y, "norm1b")
        if mlp:
            x = x + norm(routed_ff(norm(x, "norm2"), P, p + "mlp.", mlp), "norm2b")
        if cfg.get("token_side"):
            x = x + token_side(x, ids, P, p, i, cfg["token_side"]["dim"], eps)
        trail.append(x)
    z = layer_norm(x, P["final.norm"], P["final.norm.b"], eps) @ P["embed"].T * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap") or 0.0
    return (cap * torch.tanh(z / cap) if cap > 0 else z), trail
