"""Plain, slow implementation of the Kipedra decoder, written from its equations.

One function per mechanism, one sequence at a time, no cache, no batching: every quantity of a sequence is recomputed
from its token ids.  Nothing here is shared with ``tgi_b200``; the product is compared against it.  All arithmetic
happens in ``DT`` (float64 unless a caller lowers it).

Tensors are passed as a dict ``name -> torch.Tensor`` (any float dtype), the configuration as the plain dict of
``config.json``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

DT = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over the root of its mean square (last dimension), eps under the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose stored weight is the deviation from one."""
    return rms(x, eps) * (1.0 + w)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x / (1.0 + torch.exp(-x))


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def relu_squared(x: torch.Tensor) -> torch.Tensor:
    y = torch.clamp(x, min=0.0)
    return y * y


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(x, torch.zeros_like(x))


# ---- short convolution, rotation -----------------------------------------------------------------
def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u[T, C], w[C, taps]: y_t = sum over taps of w[:, j] u_{t - (taps - 1) + j}, zeros before the first token."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            y[t] += w[:, j] * padded[t + j]
    return y


def rotate_pairs(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x[T, heads, d]; token t sits at position t; dimension 2i is paired with 2i + 1, i < dims / 2."""
    y = x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


# ---- attention -----------------------------------------------------------------------------------
def sees(i: int, j: int, window: Optional[int]) -> bool:
    return j <= i and (not window or i - j < window)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: Optional[int]) -> torch.Tensor:
    """q[T, H, d], k[T, G, d], v[T, G, dv] -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(i + 1) if sees(i, j, window)]
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[i, h]) * scale
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[js, g]
    return out


def attention_inputs(h: torch.Tensor, W, p: str, mx: dict) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    rot = mx["rot"]
    q, k, v = (causal_conv(h @ W(p + n).T + W(p + n + ".b"), W(p + n + ".conv")) for n in "qkv")
    return (rotate_pairs(q.view(T, H, d), rot["dims"], rot["base"]), rotate_pairs(k.view(T, G, d), rot["dims"], rot["base"]),
            v.view(T, G, dv))


def attention(h: torch.Tensor, W, p: str, mx: dict) -> torch.Tensor:
    q, k, v = attention_inputs(h, W, p, mx)
    o = attend(q, k, v, float(mx["scale"]), mx["mask"]["size"])
    return o.reshape(h.shape[0], -1) @ W(p + "o").T


# ---- gated delta rule with one decay per head ----------------------------------------------------
def delta_scan(q, k, v, g, beta) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv], g and beta [T, H] -> o [T, H, dv]; the state starts at zero."""
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def delta(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ W(p + n).T, W(p + n + ".conv"))) for n in "qkv")
    of = [i // (H // G) for i in range(H)]
    q, k = (unit(q.view(T, G, d)) * d ** -0.5)[:, of], unit(k.view(T, G, d))[:, of]
    beta = 1.0 / (1.0 + torch.exp(-(h @ W(p + "b").T)))
    g = torch.exp(-torch.exp(W(p + "A_log")) * softplus(h @ W(p + "a").T + W(p + "dt_bias")))
    o = delta_scan(q, k, v.view(T, H, dv), g, beta)
    gate = silu(h @ W(p + "g").T).view(T, H, dv)
    return (rms(o, eps) * W(p + "norm") * gate).reshape(T, H * dv) @ W(p + "o").T


# ---- feed-forward --------------------------------------------------------------------------------
def dense(h: torch.Tensor, W, p: str) -> torch.Tensor:
    return (gelu_tanh(h @ W(p + "gate").T) * (h @ W(p + "up").T)) @ W(p + "down").T


def route(z: torch.Tensor, correction: torch.Tensor, top: int, scale: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """Router logits ``z[T, E]`` -> chosen experts and their weights, ``[T, top]`` each."""
    s = 1.0 / (1.0 + torch.exp(-z))
    chosen = torch.argsort(-(s + correction), dim=-1)[:, :top]
    w = torch.gather(s, 1, chosen)
    return chosen, w / (w.sum(dim=-1, keepdim=True) + 1e-20) * scale


def experts(h: torch.Tensor, W, p: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    chosen, w = route(h @ W(p + "router").T, W(p + "correction"), r["top"], float(r["scale"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, x in zip(chosen[t].tolist(), w[t]):
            out[t] += x * (W(f"{p}e{e}.down") @ relu_squared(W(f"{p}e{e}.up") @ h[t]))
    return out


def feed_forward(h: torch.Tensor, W, p: str, mlp: dict) -> torch.Tensor:
    return dense(h, W, p) if mlp["kind"] == "dense" else experts(h, W, p, mlp)


# ---- the model -----------------------------------------------------------------------------------
def order(cfg: dict) -> List[int]:
    """Layers in the order they run: those of the loop ``times`` times in a row."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    lo, hi = loop["start"], loop["stop"]
    return list(range(lo)) + list(range(lo, hi)) * loop["times"] + list(range(hi, n))


def block(x: torch.Tensor, W, i: int, cfg: dict) -> torch.Tensor:
    """Mixer and feed-forward side by side, both of the same stream through their own norms."""
    layer, eps, p = cfg["layers"][i], float(cfg["norm"]["eps"]), f"l{i}."
    h = norm(x, W(p + "norm1"), eps)
    y = attention(h, W, p + "mix.", layer["mixer"]) if layer["type"] == "attention" else \
        delta(h, W, p + "mix.", layer["mixer"], eps)
    if layer.get("mlp"):
        y = y + feed_forward(norm(x, W(p + "norm2"), eps), W, p + "mlp.", layer["mlp"])
    return x + float(cfg["residual_mult"]) * y


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
            dt: torch.dtype = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` collects the residual stream after every layer run."""
    dt = dt or DT
    memo: Dict[str, torch.Tensor] = {}

    def W(name):
        if name not in memo:
            memo[name] = tensors[name].to(dt)
        return memo[name]

    x = W("embed")[torch.tensor(tokens)]
    for i in order(cfg):
        x = block(x, W, i, cfg)
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, W("final.norm"), float(cfg["norm"]["eps"])) @ W("embed").T


def greedy(cfg: dict, tensors: Dict[str, torch.Tensor], prompt: List[int], new_tokens: int) -> List[int]:
    ids = list(prompt)
    for _ in range(new_tokens):
        ids.append(int(forward(cfg, tensors, ids)[-1].argmax()))
    return ids[len(prompt):]
