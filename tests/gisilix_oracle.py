"""Plain, slow implementation of the Gisilix decoder, written from its equations.

One function per mechanism, one sequence at a time, no cache, no batching: every quantity of a sequence is recomputed
from its token ids, and latent attention is computed on expanded keys and values.  Nothing here is shared with
``tgi_b200``; the product is compared against it.  All arithmetic happens in ``DT`` (float64 unless a caller lowers it).

Tensors are passed as a dict ``name -> torch.Tensor`` (any float dtype), the configuration as the plain dict of
``config.json``.
"""
from __future__ import annotations

import math
from typing import Callable, Dict, List, Optional, Tuple

import torch

DT = torch.float64


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


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


def rotate_pairs(x: torch.Tensor, rot: dict, positions: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x[T, heads, d]; token t sits at position t unless ``positions`` says otherwise; dimension 2i pairs with 2i + 1."""
    y = x.clone()
    pos = torch.arange(x.shape[0]) if positions is None else positions
    freq, amp = yarn(rot["dims"], float(rot["base"]), rot.get("scaling"))
    for i, f in enumerate(freq):
        a = pos.double() * f
        c, s = (amp * a.cos()).to(x.dtype)[:, None], (amp * a.sin()).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


# ---- attention -----------------------------------------------------------------------------------
def sees(i: int, j: int, window: Optional[int]) -> bool:
    return j <= i and (not window or i - j < window)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: Optional[int] = None,
           cap: Optional[float] = None, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q[T, H, d], k[T, G, d], v[T, G, dv] -> [T, H, dv]; ``cap`` squashes the scores, ``sink[H]`` is one more term of the
    softmax's denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    allowed = torch.tensor([[sees(i, j, window) for j in range(T)] for i in range(T)])
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        if cap:
            s = cap * torch.tanh(s / cap)
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


def temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    return 1.0 + coef * torch.log(torch.floor((positions.double() + 1.0) / every) + 1.0)


def attention_keys(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    T, G = h.shape[0], mx["kv_heads"]
    k = rms_norm(h @ W(p + "k").T, W(p + "k.norm"), eps)
    return k.view(T, G, mx["dim"]), (h @ W(p + "v").T).view(T, G, mx["vdim"])


def attention(h: torch.Tensor, kv: Tuple[torch.Tensor, torch.Tensor], W, p: str, mx: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    q = rms_norm(h @ W(p + "q").T, W(p + "q.norm"), eps).view(T, mx["heads"], mx["dim"])
    t = temperature(torch.arange(T), float(mx["q_temp"]["coef"]), mx["q_temp"]["every"])
    q = q * t.to(q.dtype)[:, None, None]
    o = attend(q, kv[0], kv[1], float(mx["scale"]), cap=float(mx["softcap"]), sink=W(p + "sink"))
    return (o.reshape(T, -1) * sigmoid(h @ W(p + "g").T)) @ W(p + "o").T


def latent_attention(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> torch.Tensor:
    """Both kinds: a rotated part, a window and a gate per head where the mixer has them."""
    T, H, d, dv, r = h.shape[0], mx["heads"], mx["dim"], mx["vdim"], mx["kv_rank"]
    rd = mx.get("rot_dim", 0)
    q = (h @ W(p + "q").T).view(T, H, d + rd)
    down = h @ W(p + "dkv").T
    c = rms_norm(down[:, :r], W(p + "dkv.norm"), eps)
    k = (c @ W(p + "uk").T).view(T, H, d)
    v = (c @ W(p + "uv").T).view(T, H, dv)
    if rd:
        shared = rotate_pairs(down[:, None, r:], mx["rot"])
        q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], mx["rot"])], dim=-1)
        k = torch.cat([k, shared.expand(T, H, rd)], dim=-1)
    o = attend(q, k, v, float(mx["scale"]), window=(mx.get("mask") or {}).get("size"))
    if rd:
        o = o * sigmoid(h @ W(p + "g").T)[:, :, None]
    return o.reshape(T, -1) @ W(p + "o").T


# ---- feed-forward --------------------------------------------------------------------------------
def dense(h: torch.Tensor, W, p: str) -> torch.Tensor:
    return (silu(h @ W(p + "gate").T) * (h @ W(p + "up").T)) @ W(p + "down").T


def route(z: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Router logits ``z[T, E]``, bias included -> chosen experts and their weights, ``[T, top]`` each."""
    chosen = torch.argsort(-z, dim=-1)[:, :top]
    zc = torch.gather(z, 1, chosen)
    e = torch.exp(zc - zc.max(dim=-1, keepdim=True).values)
    return chosen, e / e.sum(dim=-1, keepdim=True)


def experts(h: torch.Tensor, W, p: str, mlp: dict) -> torch.Tensor:
    chosen, w = route(h @ W(p + "router").T + W(p + "router.b"), mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, slot = (chosen == e).nonzero(as_tuple=True)
        out[t] += w[t, slot][:, None] * dense(h[t], W, f"{p}e{e}.")
    if mlp.get("shared"):
        out = out + dense(h, W, p + "shared.")
    return out


def feed_forward(h: torch.Tensor, W, p: str, mlp: dict) -> torch.Tensor:
    return dense(h, W, p) if mlp["kind"] == "dense" else experts(h, W, p, mlp)


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
        return layer_norm(x, W(name), W(name + ".b"), eps)

    x = W("embed")[torch.tensor(tokens)]
    kv = {}                                          # keys and values of the attention layers that have their own
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        h = norm(x, p + "norm1")
        if layer["type"] == "attention":
            src = mx.get("kv_from")
            if src is None:
                src = i
                kv[i] = attention_keys(h, W, p + "mix.", mx, eps)
            x = x + attention(h, kv[src], W, p + "mix.", mx, eps)
        else:
            x = x + latent_attention(h, W, p + "mix.", mx, eps)
        if layer.get("mlp"):
            x = x + feed_forward(norm(x, p + "norm2"), W, p + "mlp.", layer["mlp"])
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, "final.norm") @ W("embed").T


def greedy(cfg: dict, tensors: Dict[str, torch.Tensor], prompt: List[int], new_tokens: int) -> List[int]:
    ids = list(prompt)
    for _ in range(new_tokens):
        ids.append(int(forward(cfg, tensors, ids)[-1].argmax()))
    return ids[len(prompt):]
