"""Plain, slow implementation of the Sobivik decoder, written from its equations.

One function per mechanism, one sequence at a time, no cache, no batching: every quantity of a sequence is recomputed
from its token ids, latent attention is computed on expanded keys and values, retention token by token.  Nothing here is
shared with ``tgi_b200``; the product is compared against it.  All arithmetic happens in ``DT`` (float64 unless a caller
lowers it).

Tensors are passed as a dict ``name -> torch.Tensor`` (any float dtype), the configuration as the plain dict of
``config.json``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

DT = torch.float64


def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


def causal_conv(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """h[T, C], w[C, taps]: the last tap meets the token itself, the others those before it (zeros before the first)."""
    taps = w.shape[1]
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(taps):
            at = t - taps + 1 + j
            if at >= 0:
                y[t] = y[t] + w[:, j] * h[at]
    return y


def average(streams: List[torch.Tensor], w: torch.Tensor) -> torch.Tensor:
    assert len(streams) == w.numel()
    return sum(w[j] * s for j, s in enumerate(streams))


# ---- rotation ------------------------------------------------------------------------------------
def yarn(dims: int, base: float, sc: Optional[dict]) -> Tuple[List[float], float]:
    """Frequencies of the pairs and the factor on cos and sin."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / sc["factor"] * ramp + x * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x[T, heads, d]; token t sits at position t; dimension i pairs with i + dims / 2."""
    y = x.clone()
    pos, half = torch.arange(x.shape[0]), rot["dims"] // 2
    freq, amp = yarn(rot["dims"], float(rot["base"]), rot.get("scaling"))
    for i, f in enumerate(freq):
        a = pos.double() * f
        c, s = (amp * a.cos()).to(x.dtype)[:, None], (amp * a.sin()).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


# ---- attention -----------------------------------------------------------------------------------
def sees(i: int, j: int, window: Optional[int], first: int = 0) -> bool:
    return j <= i and (not window or i - j < window or j < first)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: Optional[int] = None, first: int = 0,
           sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q[T, H, d], k[T, G, d], v[T, G, dv] -> [T, H, dv]; ``first`` tokens stay visible past the window, ``sink[H]`` is one
    more term of the softmax's denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    allowed = torch.tensor([[sees(i, j, window, first) for j in range(T)] for i in range(T)])
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        s = torch.where(allowed, s, torch.full_like(s, -math.inf))
        top = s.max(dim=-1, keepdim=True).values
        if sink is not None:
            top = torch.clamp(top, min=float(sink[h]))
        e = torch.exp(s - top)
        below = e.sum(dim=-1, keepdim=True)
        if sink is not None:
            below = below + torch.exp(sink[h] - top)
        out[:, h] = (e / below) @ v[:, g]
    return out


def difference(a1: torch.Tensor, a2: torch.Tensor, lam, diff: float, eps: float) -> torch.Tensor:
    return over_rms(a1 - lam * a2, eps) * (1.0 - diff)


def strength(W, p: str, diff: float):
    return torch.exp((W(p + "lq1") * W(p + "lk1")).sum()) - torch.exp((W(p + "lq2") * W(p + "lk2")).sum()) + diff


def differential_attention(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k = (h @ W(p + "q").T).view(T, H, 2, d), (h @ W(p + "k").T).view(T, G, 2, d)
    v = (h @ W(p + "v").T).view(T, G, dv)
    mask = mx.get("mask") or {}
    maps = [attend(q[:, :, m], k[:, :, m], v, float(mx["scale"]), mask.get("size"), mask.get("keep_first", 0)) for m in range(2)]
    o = difference(maps[0], maps[1], strength(W, p, float(mx["diff"])), float(mx["diff"]), eps)
    return (o * sigmoid(h @ W(p + "g").T)[:, :, None]).reshape(T, -1) @ W(p + "o").T


def latent_attention(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> torch.Tensor:
    T, H, d, dv, r, rd = h.shape[0], mx["heads"], mx["dim"], mx["vdim"], mx["kv_rank"], mx["rot_dim"]
    cq = over_rms(h @ W(p + "dq").T, eps) * W(p + "dq.norm")
    q = (cq @ W(p + "uq").T).view(T, H, d + rd)
    down = h @ W(p + "dkv").T
    c = over_rms(down[:, :r], eps) * W(p + "dkv.norm")
    k = (c @ W(p + "uk").T).view(T, H, d)
    v = (c @ W(p + "uv").T).view(T, H, dv)
    shared = rotate_halves(down[:, None, r:], mx["rot"])
    q = torch.cat([q[..., :d], rotate_halves(q[..., d:], mx["rot"])], dim=-1)
    k = torch.cat([k, shared.expand(T, H, rd)], dim=-1)
    o = attend(q, k, v, float(mx["scale"]), window=(mx.get("mask") or {}).get("size"), sink=W(p + "sink"))
    return (o.reshape(T, -1) * sigmoid(h @ W(p + "g").T)) @ W(p + "o").T


# ---- retention -----------------------------------------------------------------------------------
def retain(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: List[float]) -> torch.Tensor:
    """q, k[T, H, d], v[T, H, dv] -> [T, H, dv]."""
    T, H, d = q.shape
    o = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=v.dtype)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h] * d ** -0.5, v[t, h])
            o[t, h] = S.T @ q[t, h]
    return o


def retention(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> torch.Tensor:
    T, H = h.shape[0], mx["heads"]
    q, k, v = ((h @ W(p + n).T).view(T, H, -1) for n in ("q", "k", "v"))
    o = over_rms(retain(q, k, v, mx["decay"]), eps)
    return (o.reshape(T, -1) * silu(h @ W(p + "g").T)) @ W(p + "o").T


MIXERS = {"retention": retention, "latent_attention": latent_attention, "attention": differential_attention}


def feed_forward(h: torch.Tensor, W, p: str) -> torch.Tensor:
    return (silu(h @ W(p + "gate").T) * (h @ W(p + "up").T)) @ W(p + "down").T


# ---- the model -----------------------------------------------------------------------------------
def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
            dt: torch.dtype = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` collects the residual stream after every layer."""
    dt, eps = dt or DT, float(cfg["norm"]["eps"])
    memo: Dict[str, torch.Tensor] = {}

    def W(name):
        if name not in memo:
            memo[name] = tensors[name].to(dt)
        return memo[name]

    def norm(x, name):
        return over_rms(x, eps) * W(name)

    x = W("embed")[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    streams = [x]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = norm(x, p + "norm1")
        h = h + causal_conv(h, W(p + "canon1"))
        x = x + norm(MIXERS[layer["type"]](h, W, p + "mix.", layer["mixer"], eps), p + "norm1b")
        if layer.get("mlp"):
            x = x + norm(feed_forward(norm(x, p + "norm2"), W, p + "mlp."), p + "norm2b")
        streams.append(x)
        x = average(streams, W(p + "dwa"))
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, "final.norm") @ W("head").T * cfg["logit_scale"]


def greedy(cfg: dict, tensors: Dict[str, torch.Tensor], prompt: List[int], new_tokens: int) -> List[int]:
    ids = list(prompt)
    for _ in range(new_tokens):
        ids.append(int(forward(cfg, tensors, ids)[-1].argmax()))
    return ids[len(prompt):]
