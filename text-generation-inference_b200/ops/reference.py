"""Plain PyTorch fp32 implementations of every op in ``tgi_b200.ops``.

They serve two purposes: they are the CPU execution path (the engine runs on a
machine without a GPU, e.g. for the tiny-Llama correctness configuration), and
they are the numerical oracle the CUDA kernels are tested against.  They favour
clarity over speed.

Tensor conventions (ragged / unpadded batches):

* ``T`` tokens of the step, ``B`` sequences, ``Hq``/``Hkv`` query/KV heads, ``D`` head size.
* KV cache of one layer: ``k_cache``/``v_cache`` of shape ``[num_blocks, block_size, Hkv, D]``;
  slot ``s`` addresses ``cache.view(-1, Hkv, D)[s]``.
* ``block_tables[B, max_blocks]`` int32; ``cu_seqlens_q[B+1]`` int32 prefix sums of the
  number of query tokens per sequence; ``kv_lens[B]`` int32 = number of KV tokens each
  sequence attends to *including* the tokens of this step.
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

FP8_MAX = 448.0
FP8 = torch.float8_e4m3fn


def rms_norm(x, residual, weight, eps: float, unit_offset: bool = False):
    if residual is not None:
        x = x + residual
    res = x
    xf = x.float()
    var = xf.pow(2).mean(-1, keepdim=True)
    y = xf * torch.rsqrt(var + eps)
    w = weight.float()
    if unit_offset:
        w = w + 1.0
    return (y * w).to(x.dtype), res


def layer_norm(x, residual, weight, bias, eps: float):
    if residual is not None:
        x = x + residual
    res = x
    y = F.layer_norm(x.float(), (x.shape[-1],), weight.float(), None if bias is None else bias.float(), eps)
    return y.to(x.dtype), res


def rotate(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, rot_dim: int, neox: bool) -> torch.Tensor:
    """Apply rotary embedding on the first ``rot_dim`` features of ``x[T, H, D]``.

    ``cos``/``sin`` are ``[T, rot_dim/2]``.  NeoX style pairs feature ``i`` with
    ``i + rot_dim/2``; GPT-J style pairs ``2i`` with ``2i+1``.
    """
    xr = x[..., :rot_dim].float()
    c = cos.float().unsqueeze(1)
    s = sin.float().unsqueeze(1)
    if neox:
        x1, x2 = xr[..., : rot_dim // 2], xr[..., rot_dim // 2 :]
        out = torch.cat([x1 * c - x2 * s, x2 * c + x1 * s], dim=-1)
    else:
        x1, x2 = xr[..., 0::2], xr[..., 1::2]
        out = torch.stack([x1 * c - x2 * s, x2 * c + x1 * s], dim=-1).flatten(-2)
    res = x.clone()
    res[..., :rot_dim] = out.to(x.dtype)
    return res


def rope_and_cache(
    qkv: torch.Tensor,
    positions: torch.Tensor,
    cos_sin: torch.Tensor,
    slots: torch.Tensor,
    k_cache: torch.Tensor,
    v_cache: torch.Tensor,
    num_heads: int,
    num_kv_heads: int,
    head_dim: int,
    rot_dim: int,
    neox: bool = True,
    k_scale: Optional[torch.Tensor] = None,
    v_scale: Optional[torch.Tensor] = None,
) -> torch.Tensor:
    """Rotate q and k inside ``qkv[T, (Hq+2Hkv)*D]``, scatter k, v into the paged cache; returns q ``[T,Hq,D]``.

    ``cos_sin[max_pos, rot_dim]`` holds ``cos`` in the first half of each row and ``sin`` in the second
    (``rot_dim == 0`` disables rotation).  For an fp8 cache the stored value is
    ``x / scale`` with a per-KV-head ``scale[Hkv]`` (``None`` means 1).
    """
    T = qkv.shape[0]
    q, k, v = qkv.split([num_heads * head_dim, num_kv_heads * head_dim, num_kv_heads * head_dim], dim=-1)
    q = q.reshape(T, num_heads, head_dim)
    k = k.reshape(T, num_kv_heads, head_dim)
    v = v.reshape(T, num_kv_heads, head_dim)
    if rot_dim > 0:
        cs = cos_sin[positions.long()]
        cos, sin = cs[:, : rot_dim // 2], cs[:, rot_dim // 2 :]
        q = rotate(q, cos, sin, rot_dim, neox)
        k = rotate(k, cos, sin, rot_dim, neox)
    kc = k_cache.view(-1, num_kv_heads, head_dim)
    vc = v_cache.view(-1, num_kv_heads, head_dim)
    idx = slots.long()
    if k_cache.dtype == FP8:
        ks = 1.0 if k_scale is None else k_scale.float().view(1, -1, 1)
        vs = 1.0 if v_scale is None else v_scale.float().view(1, -1, 1)
        # scatter through a byte view: indexed writes are not implemented for fp8 on every backend
        kc.view(torch.uint8)[idx] = (k.float() / ks).clamp(-FP8_MAX, FP8_MAX).to(FP8).view(torch.uint8)
        vc.view(torch.uint8)[idx] = (v.float() / vs).clamp(-FP8_MAX, FP8_MAX).to(FP8).view(torch.uint8)
    else:
        kc[idx] = k.to(k_cache.dtype)
        vc[idx] = v.to(v_cache.dtype)
    return q.contiguous()


def paged_attention(
    q: torch.Tensor,
    k_cache: torch.Tensor,
    v_cache: torch.Tensor,
    block_tables: torch.Tensor,
    cu_seqlens_q: torch.Tensor,
    kv_lens: torch.Tensor,
    scale: float,
    window: int = -1,
    softcap: float = 0.0,
    k_scale: Optional[torch.Tensor] = None,
    v_scale: Optional[torch.Tensor] = None,
    max_q: Optional[int] = None,
    max_kv: Optional[int] = None,
    horizon: Optional[torch.Tensor] = None,
    chunk: int = 0,
    sink=None,
    keep: int = 0,
) -> torch.Tensor:
    """Causal attention of ragged queries over paged KV (covers prefill, chunked prefill and decode).
    ``horizon[t]`` (optional) replaces the causal limit of query row ``t`` by a later position.  With ``chunk`` a row
    sees only keys ``t`` with ``t // chunk == pos // chunk``; ``sink`` adds ``exp(sink[h])`` (``True``: ``exp(0)``) to the softmax denominator.

    Query ``i`` (0-based inside its sequence's chunk of ``n`` queries) of a sequence with ``L`` KV
    tokens sits at absolute position ``L - n + i`` and attends to KV positions ``<=`` its own
    (and ``> pos - window`` when ``window > 0``).
    """
    T, Hq, D = q.shape
    nblk, bs, Hkv, _ = k_cache.shape
    group = Hq // Hkv
    Dv = v_cache.shape[3]
    out = q.new_empty(T, Hq, Dv)
    cu = cu_seqlens_q.tolist()
    lens = kv_lens.tolist()
    kc = k_cache.view(-1, Hkv, D)
    vc = v_cache.view(-1, Hkv, Dv)
    for b in range(len(lens)):
        s, e = cu[b], cu[b + 1]
        n, L = e - s, lens[b]
        if n == 0:
            continue
        nb = (L + bs - 1) // bs
        blocks = block_tables[b, :nb].long()
        slot = (blocks.unsqueeze(1) * bs + torch.arange(bs, device=q.device).unsqueeze(0)).reshape(-1)[:L]
        if kc.dtype == FP8:
            k = kc.view(torch.uint8)[slot].view(FP8).float()
            v = vc.view(torch.uint8)[slot].view(FP8).float()
        else:
            k = kc[slot].float()
            v = vc[slot].float()
        if k_scale is not None:
            k = k * k_scale.float().view(1, -1, 1)
        if v_scale is not None:
            v = v * v_scale.float().view(1, -1, 1)
        k = k.repeat_interleave(group, dim=1)  # [L, Hq, D]
        v = v.repeat_interleave(group, dim=1)
        qq = q[s:e].float()
        scores = torch.einsum("nhd,lhd->hnl", qq, k) * scale
        if softcap > 0:
            scores = softcap * torch.tanh(scores / softcap)
        qpos = torch.arange(L - n, L, device=q.device).unsqueeze(1)
        kpos = torch.arange(L, device=q.device).unsqueeze(0)
        limit = qpos if horizon is None else torch.maximum(qpos, horizon[s:e].long().clamp(max=L - 1).unsqueeze(1))
        mask = kpos <= limit
        if window > 0:
            mask &= kpos > qpos - window
        if chunk > 0:
            mask &= torch.div(kpos, chunk, rounding_mode="floor") == torch.div(qpos, chunk, rounding_mode="floor")
        if keep > 0:
            mask |= (kpos < keep) & (kpos <= limit)
        scores = scores.masked_fill(~mask.unsqueeze(0), float("-inf"))
        if sink is not None and sink is not False:
            extra = scores.new_zeros(Hq) if sink is True else sink.float()
            p = torch.softmax(torch.cat([scores, extra.view(Hq, 1, 1).expand(Hq, n, 1)], dim=-1), dim=-1)[..., :-1]
        else:
            p = torch.softmax(scores, dim=-1)
        out[s:e] = torch.einsum("hnl,lhd->nhd", p, v).to(q.dtype)
    return out


def act_and_mul(gate_up: torch.Tensor, act: str = "silu") -> torch.Tensor:
    g, u = gate_up.float().chunk(2, dim=-1)
    return (activation(g, act) * u).to(gate_up.dtype)


def activation(x: torch.Tensor, act: str) -> torch.Tensor:
    if act in ("silu", "swish"):
        return F.silu(x)
    if act in ("gelu", "gelu_python"):
        return F.gelu(x)
    if act in ("gelu_new", "gelu_fast", "gelu_pytorch_tanh", "gelu_tanh"):
        return F.gelu(x, approximate="tanh")
    if act == "relu":
        return F.relu(x)
    if act == "relu2":
        return F.relu(x).square()
    if act == "quick_gelu":
        return x * torch.sigmoid(1.702 * x)
    raise ValueError(f"unknown activation {act}")


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    return F.linear(x, weight, bias)


def embedding(ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    return F.embedding(ids.long(), table)


# ---- block-scaled fp8 -------------------------------------------------------------------------
def fp8_quant_block_weight(w: torch.Tensor, block: int = 128) -> Tuple[torch.Tensor, torch.Tensor]:
    """Quantise ``w[N,K]`` to e4m3 with one fp32 scale per ``block x block`` tile.

    Returns ``(wq[N,K] e4m3, scale[ceil(N/block), ceil(K/block)])`` with ``w ~= wq * scale``.
    """
    N, K = w.shape
    nb, kb = (N + block - 1) // block, (K + block - 1) // block
    wp = torch.zeros(nb * block, kb * block, dtype=torch.float32, device=w.device)
    wp[:N, :K] = w.float()
    tiles = wp.view(nb, block, kb, block)
    amax = tiles.abs().amax(dim=(1, 3)).clamp_min(1e-12)
    scale = amax / FP8_MAX
    q = (tiles / scale.view(nb, 1, kb, 1)).clamp(-FP8_MAX, FP8_MAX).view(nb * block, kb * block)[:N, :K]
    return q.to(FP8).contiguous(), scale.contiguous()


POW2_ACT_SCALES = False      # activation block scales rounded up to powers of two


def fp8_quant_act(x: torch.Tensor, group: int = 128) -> Tuple[torch.Tensor, torch.Tensor]:
    """Dynamic per-token, per-``group``-columns quantisation: ``x[T,K] ~= xq * scale[T, K/group]``."""
    T, K = x.shape
    assert K % group == 0
    xg = x.float().view(T, K // group, group)
    amax = xg.abs().amax(dim=-1).clamp_min(1e-12)
    scale = amax / FP8_MAX
    if POW2_ACT_SCALES:      # what the kernels do while the block-scaled MMA is in use (ops.cuda.set_fp8_mx)
        mant, expo = torch.frexp(scale)
        scale = torch.where(mant == 0.5, scale, torch.ldexp(torch.ones_like(scale), expo))
    q = (xg / scale.unsqueeze(-1)).clamp(-FP8_MAX, FP8_MAX).view(T, K)
    return q.to(FP8), scale.contiguous()


def fp8_dequant_block_weight(wq: torch.Tensor, scale: torch.Tensor, block: int = 128) -> torch.Tensor:
    N, K = wq.shape
    s = scale.repeat_interleave(block, 0)[:N].repeat_interleave(block, 1)[:, :K]
    return wq.float() * s


def gemm_fp8_block(
    xq: torch.Tensor,
    xs: torch.Tensor,
    wq: torch.Tensor,
    ws: torch.Tensor,
    out_dtype: torch.dtype = torch.bfloat16,
    bias: Optional[torch.Tensor] = None,
    block: int = 128,
) -> torch.Tensor:
    """``out[T,N] = (xq*xs) @ (wq*ws)^T`` with 1x128 activation and 128x128 weight scales."""
    x = xq.float() * xs.repeat_interleave(block, dim=1)[:, : xq.shape[1]]
    w = fp8_dequant_block_weight(wq, ws, block)
    out = x @ w.t()
    if bias is not None:
        out = out + bias.float()
    return out.to(out_dtype)


def fp8_quant_per_tensor(x: torch.Tensor, scale: Optional[torch.Tensor] = None, scale_ub: Optional[float] = None):
    """Per-tensor e4m3 quantisation; dynamic when ``scale`` is None."""
    if scale is None:
        amax = x.abs().max().float()
        if scale_ub is not None:
            amax = amax.clamp(max=scale_ub)
        scale = (amax / FP8_MAX).clamp_min(1e-12)
    q = (x.float() / scale).clamp(-FP8_MAX, FP8_MAX).to(FP8)
    return q, scale.reshape(()).float()


# ---- sampling ---------------------------------------------------------------------------------
def argmax_logprob(logits: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """Greedy token and its log-probability for each row of ``logits[B,V]``."""
    lp = torch.log_softmax(logits.float(), dim=-1)
    ids = lp.argmax(dim=-1)
    return ids, lp.gather(1, ids.unsqueeze(1)).squeeze(1)


# ---- MoE --------------------------------------------------------------------------------------
def moe_topk_softmax(router_logits: torch.Tensor, top_k: int, renormalize: bool = True):
    probs = torch.softmax(router_logits.float(), dim=-1)
    w, idx = torch.topk(probs, top_k, dim=-1)
    if renormalize:
        w = w / w.sum(dim=-1, keepdim=True)
    return w, idx


def moe_route_sigmoid(x, weight, correction, top_k: int, scale: float):
    s = torch.sigmoid(F.linear(x.float(), weight.float()))
    idx = torch.topk(s + correction, top_k, dim=-1)[1]
    w = s.gather(1, idx)
    return w / (w.sum(-1, keepdim=True) + 1e-20) * scale, idx


def moe_route_softmax(x, weight, bias, top_k: int):
    z, idx = torch.topk(F.linear(x.float(), weight.float(), bias), top_k, dim=-1)
    return torch.softmax(z, dim=-1), idx


def moe_plain_experts(x, w_up, w_down, topk_weights, topk_ids, act: str, gated: bool = False):
    """``w_up[E, I, H]``, ``w_down[E, H, I]``: sum over a token's experts of weight times ``down(act(up x))``."""
    if gated:
        return moe_experts(x, w_up, w_down, topk_weights, topk_ids, act)
    out = torch.zeros(x.shape, dtype=torch.float32, device=x.device)
    for e in range(w_up.shape[0]):
        tok, slot = (topk_ids == e).nonzero(as_tuple=True)
        if tok.numel():
            y = F.linear(activation(F.linear(x[tok], w_up[e]), act), w_down[e]).float()
            out.index_add_(0, tok, y * topk_weights[tok, slot].unsqueeze(1).float())
    return out.to(x.dtype)


def moe_sparsemixer(router_logits: torch.Tensor, jitter_eps: float = 0.01) -> Tuple[torch.Tensor, torch.Tensor]:
    """Top-2 routing of Phi-3.5-MoE ("sparsemixer", inference form): each of the two picks is the arg-max of
    the remaining logits, and its weight is the softmax over the logits that lie within a relative
    band ``2 * jitter_eps`` of that maximum."""
    s = router_logits.float()
    neg = float("-inf")
    m1, i1 = s.max(-1, keepdim=True)
    mask1 = ((m1 - s) / s.abs().clamp(min=m1)) > 2 * jitter_eps
    g1 = torch.softmax(s.masked_fill(mask1, neg), -1).gather(-1, i1)
    s2 = s.scatter(-1, i1, neg)
    m2, i2 = s2.max(-1, keepdim=True)
    mask2 = ((m2 - s) / s.abs().clamp(min=m2)) > 2 * jitter_eps
    g2 = torch.softmax(s2.masked_fill(mask2, neg), -1).gather(-1, i2)
    return torch.cat([g1, g2], -1), torch.cat([i1, i2], -1)


def moe_experts(
    x: torch.Tensor,
    w_gate_up: torch.Tensor,
    w_down: torch.Tensor,
    topk_weights: torch.Tensor,
    topk_ids: torch.Tensor,
    act: str = "silu",
    first: int = 0,
) -> torch.Tensor:
    """Dense-loop mixture of experts: ``w_gate_up[E, 2I, H]``, ``w_down[E, H, I]`` hold the experts
    ``first .. first + E - 1``; slots routed to other experts contribute nothing."""
    T, H = x.shape
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    E = w_gate_up.shape[0]
    for e in range(E):
        tok, slot = (topk_ids == e + first).nonzero(as_tuple=True)
        if tok.numel() == 0:
            continue
        h = F.linear(x[tok], w_gate_up[e])
        h = act_and_mul(h, act)
        y = F.linear(h, w_down[e]).float()
        out.index_add_(0, tok, y * topk_weights[tok, slot].unsqueeze(1).float())
    return out.to(x.dtype)


# ---- token mixers of hybrid decoders -------------------------------------------------------------
def embed_residual(ids, table, scale: float = 1.0, streams: int = 1):
    x = F.embedding(ids.long(), table).float() * scale
    return x if streams == 1 else torch.cat([x.unsqueeze(0), x.new_zeros(streams - 1, *x.shape)])


def stream_step(delta, post, residual, weight, eps: float, rows=None, keep: bool = True, gain: float = 1.0, average=None, streams=None,
                conv=None):
    r = residual
    if delta is not None:
        r = r + (delta.float() if post is None else _row_rms(delta, post.float(), eps))
    if average is not None:
        n = average.shape[0]
        r = torch.einsum("n,nth->th", average, torch.cat([streams[:n - 1], r.unsqueeze(0)])) if rows is not None else _averaged(streams, r, average)
    if rows is not None:
        r = r[rows.long()]
    out = (_row_rms(r, weight.float(), eps) * gain).to(weight.dtype)
    return (out if conv is None else input_conv(out, conv)), r if keep else None


def _averaged(streams, r, average):
    n = average.shape[0]
    streams[n - 1] = r
    return torch.einsum("n,nth->th", average, streams[:n])


def input_conv(x, conv):
    return _conv_rows(x, (0,), (x.shape[1],), conv.weights, conv.cu, conv.kv_lens, conv.state_slots, conv.state).to(x.dtype)


def residual_norm(delta, residual, weight, eps: float, rows=None, keep: bool = True, scale: float = 1.0,
                  unit_offset: bool = False, weight2=None, layer: bool = False, bias=None):
    r = residual
    if delta is not None:
        parts = delta if isinstance(delta, tuple) else (delta,)
        r = residual + scale * sum(d.float() for d in parts)
    if rows is not None:
        r = r[rows.long()]
    d = r - r.mean(-1, keepdim=True) if layer else r
    x = d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + eps)
    b = 0.0 if bias is None else bias.float()
    ys = tuple((x * (w.float() + (1.0 if unit_offset else 0.0)) + b).to(w.dtype) for w in (weight, weight2) if w is not None)
    return ys + (r if keep else None,)


def _sequences(cu, kv_lens, state_slots):
    """``(sequence, first row, rows, position of the first row, slot)`` of every sequence that brings tokens."""
    cu, lens, slots = cu.tolist(), kv_lens.tolist(), state_slots.tolist()
    for b, (s, e) in enumerate(zip(cu[:-1], cu[1:])):
        if e > s:
            yield b, s, e - s, lens[b] - (e - s), slots[b]


def _short_conv(x, w, past):
    """``x[n, C]`` after ``past[taps - 1, C]``; returns the convolved rows and the new past."""
    taps = w.shape[0]
    full = torch.cat([past.float(), x.float()], dim=0)
    y = sum(full[j:j + x.shape[0]] * w[j].float() for j in range(taps))
    return y, full[full.shape[0] - (taps - 1):]


def _conv_rows(proj, offs, widths, conv_t, cu, kv_lens, state_slots, conv_state):
    """Column groups ``offs`` / ``widths`` of ``proj`` side by side after their short convolutions, fp32; advances
    ``conv_state``."""
    x = torch.cat([proj[:, o:o + w] for o, w in zip(offs, widths)], dim=1)
    taps = conv_state.shape[1] + 1
    w = conv_t[conv_t.shape[0] - taps:]
    y = torch.zeros(x.shape)
    for _, s, n, start, slot in _sequences(cu, kv_lens, state_slots):
        past = conv_state[slot] if slot >= 0 and start > 0 else torch.zeros(taps - 1, x.shape[1])
        y[s:s + n], new = _short_conv(x[s:s + n], w, past)
        if slot >= 0:
            conv_state[slot] = new.to(conv_state.dtype)
    return y


def rotate_norm_store(proj, offs, positions, cos_sin, slots, k_cache, v_cache, num_heads, num_kv_heads, dim, vdim, rot_dim,
                      qk_norm, eps, v_first=None, v_lambda: float = 0.0, interleaved: bool = False, conv=None):
    T = proj.shape[0]
    if conv is not None:
        widths = (num_heads * dim, num_kv_heads * dim, num_kv_heads * vdim)
        proj_dtype, proj = proj.dtype, _conv_rows(proj, offs, widths, conv.weights, conv.cu, conv.kv_lens, conv.state_slots,
                                                  conv.state)
        offs = (0, widths[0], widths[0] + widths[1])
    else:
        proj_dtype = proj.dtype
    cs = cos_sin[positions.long()]
    cos, sin = cs[:, : rot_dim // 2], cs[:, rot_dim // 2:]

    def head(off, n):
        x = proj[:, off:off + n * dim].reshape(T, n, dim).float()
        if rot_dim > 0:
            x = rotate(x, cos, sin, rot_dim, not interleaved)
        return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) if qk_norm else x

    q, k = head(offs[0], num_heads), head(offs[1], num_kv_heads)
    v = proj[:, offs[2]:offs[2] + num_kv_heads * vdim].float()
    if v_first is not None:
        v = (1.0 - v_lambda) * v + v_lambda * v_first.float()
    ok = (slots >= 0).nonzero(as_tuple=True)[0]
    idx = slots[ok].long()
    k_cache.view(-1, num_kv_heads, k_cache.shape[3])[idx, :, :dim] = k[ok].to(k_cache.dtype)
    v_cache.view(-1, num_kv_heads, v_cache.shape[3])[idx, :, :vdim] = v.view(T, num_kv_heads, vdim)[ok].to(v_cache.dtype)
    return F.pad(q, (0, k_cache.shape[3] - dim)).to(proj_dtype)


def _store_rows(pages, slots, rows, col: int = 0):
    """``rows[T, heads, n]`` to columns ``col ..`` of the tokens' slots."""
    ok = (slots >= 0).nonzero(as_tuple=True)[0]
    flat = pages.view(-1, pages.shape[2], pages.shape[3])
    flat[slots[ok].long(), :, col:col + rows.shape[2]] = rows[ok].to(pages.dtype)


def _row_rms(x, weight, eps: float):
    x = x.float()
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight


def row_norm_store(proj, offs, positions, slots, k_cache, v_cache, q_weight, k_weight, eps: float, num_heads, num_kv_heads, dim,
                   vdim, width, temperature=None):
    T = proj.shape[0]
    q = _row_rms(proj[:, offs[0]:offs[0] + num_heads * dim], q_weight, eps)
    if temperature is not None:
        coef, every = temperature
        q = q * (1.0 + coef * torch.log(torch.div(positions + 1, every, rounding_mode="floor").float() + 1.0)).unsqueeze(1)
    if k_weight is not None:
        k = _row_rms(proj[:, offs[1]:offs[1] + num_kv_heads * dim], k_weight, eps)
        _store_rows(k_cache, slots, k.view(T, num_kv_heads, dim))
        _store_rows(v_cache, slots, proj[:, offs[2]:offs[2] + num_kv_heads * vdim].reshape(T, num_kv_heads, vdim))
    return F.pad(q.view(T, num_heads, dim), (0, width - dim)).to(proj.dtype)


def map_store(proj, offs, slots, k_cache, v_cache, num_heads: int, num_kv_heads: int, dim: int, vdim: int):
    T = proj.shape[0]
    part = lambda i, n: proj[:, offs[i]:offs[i] + n]
    _store_rows(k_cache, slots, part(1, num_kv_heads * 2 * dim).reshape(T, num_kv_heads, 2 * dim))
    _store_rows(v_cache, slots, part(2, num_kv_heads * vdim).reshape(T, num_kv_heads, vdim))
    q = proj.new_zeros(T, num_heads, 2, k_cache.shape[3])
    maps = part(0, num_heads * 2 * dim).reshape(T, num_heads, 2, dim)
    for m in range(2):
        q[:, :, m, m * dim:(m + 1) * dim] = maps[:, :, m]
    return q.view(T, 2 * num_heads, -1)


def map_difference(a, gate, lam: float, factor: float, eps: float, width: int):
    T = a.shape[0]
    x = a[..., :width].float()
    y = _row_rms(x[:, 0::2] - lam * x[:, 1::2], factor, eps)
    if gate is not None:
        y = y * torch.sigmoid(gate.float()).unsqueeze(2)
    return y.reshape(T, -1).to(a.dtype)


def output_gate(x, gate, width: int):
    T = x.shape[0]
    return (x[:, :, :width].reshape(T, -1).float() * torch.sigmoid(gate.float())).to(x.dtype)


def latent_store(proj, off_c, weight, eps: float, positions, cos_sin, slots, pages, q, off_rot, rank, rot, heads, dim,
                 q_full=None, queries: bool = True, q_latent=None, width=None):
    assert q_full is None
    T = proj.shape[0]
    cs = cos_sin[positions.long()]
    turn = lambda x: rotate(x.float(), cs[:, :rot // 2], cs[:, rot // 2:], rot, False)
    if pages is not None:
        _store_rows(pages, slots, _row_rms(proj[:, off_c:off_c + rank], weight, eps).unsqueeze(1))
    if pages is not None and rot:
        _store_rows(pages, slots, turn(proj[:, off_c + rank:off_c + rank + rot].unsqueeze(1)), off_rot)
    if q_latent is not None:
        off, w, out = q_latent
        out.copy_(F.pad(_row_rms(proj[:, off:off + w.shape[0]], w, eps), (0, out.shape[1] - w.shape[0])))
    if queries and rot:
        q[:, :, off_rot:off_rot + rot] = turn(proj[:, :heads * (dim + rot)].reshape(T, heads, dim + rot)[..., dim:]).to(q.dtype)


def latent_attention(q, pages, rank, block_tables, cu_seqlens_q, kv_lens, scale: float, window: int = -1, max_q=None, max_kv=None,
                     gate=None, elsewhere=None, sink=None):
    assert elsewhere is None
    o = paged_attention(q, pages, pages[..., :rank].contiguous(), block_tables, cu_seqlens_q, kv_lens, scale, window, sink=sink)
    return o if gate is None else (o.float() * torch.sigmoid(gate.float()).unsqueeze(2)).to(o.dtype)


def delta_inputs(proj, offs, a_pre, conv_t, a_log, dt_bias, cu, kv_lens, state_slots, conv_state, kv_heads, heads, dim,
                 pitch, vdim, single: bool, head_decay: bool = False):
    T = proj.shape[0]
    nq, nv = kv_heads * dim, heads * vdim
    y = F.silu(_conv_rows(proj, offs, (nq, nq, nv), conv_t, cu, kv_lens, state_slots, conv_state))
    q, k = (y[:, i * nq:(i + 1) * nq].view(T, kv_heads, dim) for i in range(2))
    q = q * torch.rsqrt(q.pow(2).sum(-1, keepdim=True) + 1e-6) * dim ** -0.5
    k = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
    step = F.softplus(a_pre.float() + dt_bias).view(T, heads, 1 if head_decay else dim)
    g = torch.exp(-torch.exp(a_log).view(1, heads, 1) * step)
    beta = torch.sigmoid(proj[:, offs[3]:offs[3] + heads].float())
    pad = (0, pitch - dim)
    g = g.squeeze(2) if head_decay else F.pad(g, pad)
    return F.pad(q, pad), F.pad(k, pad), y[:, 2 * nq:].view(T, heads, vdim), g, beta, (q * k).sum(-1)


def delta_scan(q, k, v, g, beta, qk, cu, kv_lens, state_slots, state, dim: int, max_q: int):
    T, heads, vdim = v.shape
    rep = heads // k.shape[1]
    q, k = q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1)
    out = torch.zeros(T, heads, vdim)
    for _, s, n, start, slot in _sequences(cu, kv_lens, state_slots):
        S = state[slot].clone() if slot >= 0 and start > 0 else torch.zeros(state.shape[1:])      # [H, vdim, pitch]
        for t in range(s, s + n):
            S = S * g[t].view(heads, 1, -1)
            u = beta[t].unsqueeze(1) * (v[t] - torch.einsum("hvd,hd->hv", S, k[t]))
            S = S + u.unsqueeze(2) * k[t].unsqueeze(1)
            out[t] = torch.einsum("hvd,hd->hv", S, q[t])
        if slot >= 0:
            state[slot] = S
    return out


def decay_scan(proj, offs, decay, cu, kv_lens, state_slots, state, heads: int, dim: int, vdim: int, max_q: int,
               act: str = "silu", k_scale: float = 1.0):
    T = proj.shape[0]
    fn = F.silu if act else (lambda x: x)
    q, k = (fn(proj[:, o:o + heads * dim].float()).reshape(T, heads, dim) for o in offs[:2])
    v = fn(proj[:, offs[2]:offs[2] + heads * vdim].float()).reshape(T, heads, vdim)
    k = k * k_scale
    pad = (0, state.shape[3] - dim)
    q, k = F.pad(q, pad), F.pad(k, pad)
    out = torch.zeros(T, heads, vdim)
    for _, s, n, start, slot in _sequences(cu, kv_lens, state_slots):
        S = state[slot].clone() if slot >= 0 and start > 0 else torch.zeros(state.shape[1:])
        for t in range(s, s + n):
            S = S * decay.view(-1, 1, 1) + v[t].unsqueeze(2) * k[t].unsqueeze(1)
            out[t] = torch.einsum("hvd,hd->hv", S, q[t])
        if slot >= 0:
            state[slot] = S
    return out


def gated_norm(o, gate, weight, eps: float, groups: int, out_cols: int, act: str = "sigmoid"):
    T = o.shape[0]
    x = o.reshape(T, groups, -1)
    y = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight
    fn = torch.sigmoid if act == "sigmoid" else F.silu
    y = y.reshape(T, -1) * fn(gate[:, :y.shape[1] * y.shape[2]].float())
    return F.pad(y, (0, out_cols - y.shape[1])).to(gate.dtype)
