"""Plain, slow implementation of the Fuzuvik decoder, written from its equations.

One function per mechanism, one sequence at a time, no cache, no batching: every quantity of a sequence is
recomputed from its token ids.  Nothing here is shared with ``tgi_b200``; the product is compared against it.
All arithmetic happens in ``DT`` (float64 unless a caller lowers it).

Tensors are passed as a dict ``name -> torch.Tensor`` (any float dtype), the configuration as the plain dict of
``config.json``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

DT = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over the root of its mean square (last dimension), eps under the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_erf(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


# ---- rotary --------------------------------------------------------------------------------------
def frequencies(rot: dict) -> List[float]:
    """Angular frequency of every rotated pair, after the wavelength-dependent rescaling."""
    n = int(rot["dims"])
    sc = rot.get("scaling")
    out = []
    for i in range(n // 2):
        f = float(rot["base"]) ** (-2.0 * i / n)
        if sc:
            wave = 2.0 * math.pi / f
            if wave < sc["original"] / sc["high"]:
                pass
            elif wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            else:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x[T, heads, dim]; token t sits at position t; dimension i is paired with i + dims / 2."""
    n = int(rot["dims"])
    half = n // 2
    y = x.clone()
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(frequencies(rot), dtype=torch.float64)[None]
    c, s = ang.cos().to(x.dtype)[:, None], ang.sin().to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:n]
    y[..., :half] = u * c - v * s
    y[..., half:n] = v * c + u * s
    return y


# ---- attention -----------------------------------------------------------------------------------
def sees(i: int, j: int, chunk: Optional[int]) -> bool:
    return j <= i and (not chunk or i // chunk == j // chunk)


def sink_softmax(scores: torch.Tensor) -> torch.Tensor:
    """exp(s) over (1 + sum of exp(s)): one more key of score 0 that carries no value."""
    m = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(scores - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, chunk: Optional[int]) -> torch.Tensor:
    """q[T, H, d], k[T, G, d], v[T, G, dv] -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(i + 1) if sees(i, j, chunk)]
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[i, h]) * scale
            out[i, h] = sink_softmax(s) @ v[js, g]
    return out


def attention(h: torch.Tensor, W, p: str, mx: dict, eps: float, first: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = rms(rotate((h @ W(p + "q").T).view(T, H, d), mx["rot"]), eps)
    k = rms(rotate((h @ W(p + "k").T).view(T, G, d), mx["rot"]), eps)
    v = (h @ W(p + "v").T).view(T, G, dv)
    if mx.get("v_mix"):
        if "v" not in first:
            first["v"] = v
        else:
            lam = W(p + "vmix").reshape(())
            v = (1 - lam) * v + lam * first["v"]
    mask = mx.get("mask") or {}
    o = attend(q, k, v, float(mx["scale"]), mask.get("size"))
    return o.reshape(T, H * dv) @ W(p + "o").T


# ---- gated delta rule with one decay per key channel ---------------------------------------------
def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x[T, C], w[C, taps]; the last tap belongs to the token itself, the past before token 0 is zero."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1 - j)
            if src >= 0:
                y[t] += w[:, j] * x[src]
    return y


def delta_scan(q, k, v, g, beta) -> torch.Tensor:
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H] -> o [T, H, dv]; the state starts at zero."""
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def channel_delta(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = silu(causal_conv(h @ W(p + "q").T, W(p + "q.conv"))).view(T, G, d)
    k = silu(causal_conv(h @ W(p + "k").T, W(p + "k.conv"))).view(T, G, d)
    v = silu(causal_conv(h @ W(p + "v").T, W(p + "v.conv"))).view(T, H, dv)
    of = [i // (H // G) for i in range(H)]
    q, k = (unit(q) * d ** -0.5)[:, of], unit(k)[:, of]
    beta = torch.sigmoid(h @ W(p + "b").T)
    step = torch.nn.functional.softplus((h @ W(p + "a1").T) @ W(p + "a2").T + W(p + "dt_bias")).view(T, H, d)
    g = torch.exp(-torch.exp(W(p + "A_log"))[None, :, None] * step)
    o = delta_scan(q, k, v, g, beta)
    gate = torch.sigmoid((h @ W(p + "g1").T) @ W(p + "g2").T).view(T, H, dv)
    return (rms(o, eps) * W(p + "norm") * gate).reshape(T, H * dv) @ W(p + "o").T


# ---- linear attention with one fixed decay per head ----------------------------------------------
def lightning_scan(q, k, v, decay) -> torch.Tensor:
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    lam = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = lam * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def lightning(h: torch.Tensor, W, p: str, mx: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
    q, k = silu(h @ W(p + "q").T).view(T, H, d), silu(h @ W(p + "k").T).view(T, H, d)
    v = silu(h @ W(p + "v").T).view(T, H, dv)
    o = lightning_scan(q, k, v, mx["decay"]).reshape(T, H * dv)
    return (rms(o, eps) * W(p + "norm") * torch.sigmoid(h @ W(p + "g").T)) @ W(p + "o").T


# ---- the model -----------------------------------------------------------------------------------
def feed_forward(h: torch.Tensor, W, p: str, mlp: dict) -> torch.Tensor:
    assert mlp["kind"] == "dense"
    return gelu_erf(h @ W(p + "up").T) @ W(p + "down").T


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
            dt: torch.dtype = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` collects the residual stream after every layer."""
    dt = dt or DT
    memo: Dict[str, torch.Tensor] = {}

    def W(name):
        if name not in memo:
            memo[name] = tensors[name].to(dt)
        return memo[name]

    eps = float(cfg["norm"]["eps"])
    x = W("embed")[torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    first: dict = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        h = rms(x, eps) * W(p + "norm1")
        if layer["type"] == "attention":
            m = attention(h, W, p + "mix.", mx, eps, first)
        elif layer["type"] == "channel_delta":
            m = channel_delta(h, W, p + "mix.", mx, eps)
        elif layer["type"] == "lightning":
            m = lightning(h, W, p + "mix.", mx, eps)
        else:
            raise ValueError(layer["type"])
        x = x + m
        if layer.get("mlp"):
            x = x + feed_forward(rms(x, eps) * W(p + "norm2"), W, p + "mlp.", layer["mlp"])
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * W("final.norm")) @ W("head").T


def greedy(cfg: dict, tensors: Dict[str, torch.Tensor], prompt: List[int], new_tokens: int) -> List[int]:
    ids = list(prompt)
    for _ in range(new_tokens):
        ids.append(int(forward(cfg, tensors, ids)[-1].argmax()))
    return ids[len(prompt):]
