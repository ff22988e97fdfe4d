"""Op front end: routes every hot op to the sm_100a kernels (CUDA tensors) or the PyTorch oracle (CPU).

On a CUDA tensor the native kernel library is *required*: if it has not been
built, the call raises instead of silently running a PyTorch fallback.  Setting
``TGI_B200_OPS=torch`` selects the PyTorch implementations on the GPU as well;
that switch exists for A/B numerics checks and for the library-kernel baseline
path, never as a default.
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Optional

import torch

from . import reference as ref

_FORCE_TORCH = os.environ.get("TGI_B200_OPS", "") == "torch"
_backend = None


def native():
    """The CUDA kernel backend module (loads the in-tree shared library on first use)."""
    global _backend
    if _backend is None:
        from . import cuda as _cuda_backend

        _cuda_backend.load()
        _backend = _cuda_backend
    return _backend


def use_native(t: torch.Tensor) -> bool:
    return t.is_cuda and not _FORCE_TORCH


def set_force_torch(flag: bool) -> None:
    global _FORCE_TORCH
    _FORCE_TORCH = flag


def rms_norm(x, residual, weight, eps, unit_offset=False):
    if use_native(x):
        return native().rms_norm(x, residual, weight, eps, unit_offset)
    return ref.rms_norm(x, residual, weight, eps, unit_offset)


def rms_norm_quant(x, residual, weight, eps, unit_offset=False):
    """Residual-add + RMSNorm + 1x128 e4m3 quantisation: returns ``(xq, scales, new_residual)``."""
    if use_native(x):
        return native().rms_norm_quant(x, residual, weight, eps, unit_offset)
    y, res = ref.rms_norm(x, residual, weight, eps, unit_offset)
    q, s = ref.fp8_quant_act(y)
    return q, s, res


def layer_norm(x, residual, weight, bias, eps):
    if use_native(x):
        return native().layer_norm(x, residual, weight, bias, eps)
    return ref.layer_norm(x, residual, weight, bias, eps)


def rope_and_cache(qkv, positions, cos_sin, slots, k_cache, v_cache, num_heads, num_kv_heads, head_dim,
                   rot_dim, neox=True, k_scale=None, v_scale=None):
    if use_native(qkv):
        return native().rope_and_cache(qkv, positions, cos_sin, slots, k_cache, v_cache, num_heads,
                                       num_kv_heads, head_dim, rot_dim, neox, k_scale, v_scale)
    return ref.rope_and_cache(qkv, positions, cos_sin, slots, k_cache, v_cache, num_heads, num_kv_heads,
                              head_dim, rot_dim, neox, k_scale, v_scale)


def paged_attention(q, k_cache, v_cache, block_tables, cu_seqlens_q, kv_lens, scale, window=-1, softcap=0.0,
                    k_scale=None, v_scale=None, max_q=None, max_kv=None, horizon=None, chunk=0, sink=None, keep=0):
    """``horizon`` (optional int32 ``[T]``): last KV position each query row may see when that is past its own
    position (image rows that attend to their whole image); ``None`` is plain causal attention.  ``chunk`` > 0: rows see
    only keys of their own chunk of ``chunk`` positions.  ``sink``: one more key without a value in the softmax, of the score
    given per head (fp32 ``[Hq]``; ``True``: 0), which is neither scaled nor capped.  ``keep``: the first tokens of a sequence,
    visible whatever the window."""
    if use_native(q):
        return native().paged_attention(q, k_cache, v_cache, block_tables, cu_seqlens_q, kv_lens, scale,
                                        window, softcap, k_scale, v_scale, max_q, max_kv, horizon=horizon, chunk=chunk, sink=sink, keep=keep)
    return ref.paged_attention(q, k_cache, v_cache, block_tables, cu_seqlens_q, kv_lens, scale, window,
                               softcap, k_scale, v_scale, horizon=horizon, chunk=chunk, sink=sink, keep=keep)


def act_and_mul(gate_up, act="silu"):
    if use_native(gate_up):
        return native().act_and_mul(gate_up, act)
    return ref.act_and_mul(gate_up, act)


def act_and_mul_quant(gate_up, act="silu"):
    """``act(gate) * up`` followed by 1x128 e4m3 quantisation: ``(q, scales)``."""
    if use_native(gate_up):
        return native().act_and_mul_quant(gate_up, act)
    return ref.fp8_quant_act(ref.act_and_mul(gate_up, act))


def activation(x, act):
    if use_native(x) and x.dtype in (torch.bfloat16, torch.float32) and x.is_contiguous():
        return native().activation(x, act)
    return ref.activation(x, act)


# ---- token mixers of hybrid decoders -------------------------------------------------------------
def _mixer_backend(t):
    return native() if use_native(t) else ref


def embed_residual(ids, table, scale=1.0, streams=1):
    """``table[ids] * scale`` as the fp32 residual stream ``[T, H]``; with ``streams`` > 1 as the first of so many,
    ``[streams, T, H]``, the others not yet written."""
    return _mixer_backend(table).embed_residual(ids, table, scale, streams)


def stream_step(delta, post, residual, weight, eps, rows=None, keep=True, gain=1.0, average=None, streams=None, conv=None):
    """``r = residual + RMSNorm(delta) * post`` in fp32 (``post`` ``None``: plus ``delta``; ``delta`` ``None``: ``residual``).  With
    ``average`` (fp32 ``[n]``), ``r`` is kept as ``streams[n - 1]`` and replaced by the sum over ``streams[:n]`` so weighted.
    Returns ``(RMSNorm(r) * weight * gain, r)`` as ``residual_norm`` does; ``rows`` and ``keep`` as there (chosen rows are not
    kept in ``streams``).  ``conv`` (a ``ShortConv`` of all columns): what comes out is convolved over time."""
    backend = _mixer_backend(residual)
    inside = conv is not None and conv.single
    out, r = backend.stream_step(delta, post, residual, weight, eps, rows, keep, gain, average, streams, conv if inside else None)
    return (out if conv is None or inside else backend.input_conv(out, conv)), r


def residual_norm(delta, residual, weight, eps, rows=None, keep=True, scale=1.0, unit_offset=False, weight2=None, layer=False,
                  bias=None):
    """``r = residual + scale * delta`` in fp32 (``delta``: a tensor, a pair whose sum it is, or ``None``) and
    ``RMSNorm(r) * weight`` (``unit_offset``: times ``1 + weight``; ``layer``: of ``r`` minus its mean; plus ``bias``) in the
    weight's dtype: ``(normed, r)``, with ``weight2`` ``(normed, normed by weight2, r)``.  ``rows`` picks the rows to compute;
    ``keep=False`` drops ``r``."""
    return _mixer_backend(residual).residual_norm(delta, residual, weight, eps, rows, keep, scale, unit_offset, weight2, layer,
                                                  bias)


@dataclass
class ShortConv:
    """Causal convolution over time of a step's q, k and v: weights (``conv_weights``), the pool of past inputs
    ``[slots, taps - 1, channels]``, and which sequence brings which rows.  ``single``: one token per sequence at most."""

    weights: torch.Tensor
    state: torch.Tensor
    cu: torch.Tensor
    kv_lens: torch.Tensor
    state_slots: torch.Tensor
    single: bool


def attention_pitch(dim, vdim, dtype, device):
    """Page widths of a head's keys and values on ``device`` (see ``ops.cuda.attention_pitch``)."""
    if torch.device(device).type == "cuda" and not _FORCE_TORCH:
        return native().attention_pitch(dim, vdim, dtype)
    return dim, vdim


def rotate_norm_store(proj, offs, positions, cos_sin, slots, k_cache, v_cache, num_heads, num_kv_heads, dim, vdim, rot_dim,
                      qk_norm, eps, v_first=None, v_lambda=0.0, interleaved=False, conv=None):
    """``proj[T, *]`` with q, k, v from columns ``offs``: convolve all three over time (``conv``, a ``ShortConv``), rotate
    q and k (pairs ``i, i + rot_dim / 2``, or ``2i, 2i + 1`` when ``interleaved``), divide them by their root mean square
    per head (``qk_norm``), mix v with ``v_first`` (``(1 - lambda) v + lambda v_first``), store k and v; returns q
    ``[T, Hq, Dk]``."""
    return _mixer_backend(proj).rotate_norm_store(proj, offs, positions, cos_sin, slots, k_cache, v_cache, num_heads,
                                                  num_kv_heads, dim, vdim, rot_dim, qk_norm, eps, v_first, v_lambda,
                                                  interleaved, conv)


def row_norm_store(proj, offs, positions, slots, k_cache, v_cache, q_weight, k_weight, eps, num_heads, num_kv_heads, dim, vdim,
                   width, temperature=None):
    """``proj[T, *]`` with q, k, v from columns ``offs``: q and k over the root mean square of their whole rows, times their
    weights; q times ``1 + coef * ln(floor((position + 1) / every) + 1)`` (``temperature = (coef, every)``); k and v stored
    (``k_weight`` ``None``: the layer has queries only).  Returns q ``[T, Hq, width]``, zeros past ``dim``."""
    return _mixer_backend(proj).row_norm_store(proj, offs, positions, slots, k_cache, v_cache, q_weight, k_weight, eps, num_heads,
                                               num_kv_heads, dim, vdim, width, temperature)


def map_store(proj, offs, slots, k_cache, v_cache, num_heads, num_kv_heads, dim, vdim):
    """``proj[T, *]`` with q and k (two maps of ``dim`` per head) and v from columns ``offs``: k and v stored, the maps of a key
    head side by side.  Returns ``[T, 2 Hq, Dk]``: every query map alone at its place in such a row, zeros elsewhere."""
    return _mixer_backend(proj).map_store(proj, offs, slots, k_cache, v_cache, num_heads, num_kv_heads, dim, vdim)


def map_difference(a, gate, lam, factor, eps, width):
    """``a[T, 2 H, pitch]``: even rows minus ``lam`` times odd rows, over their root mean square (first ``width`` columns), times
    ``factor`` and ``sigmoid(gate[T, H])`` (``None``: no gate); ``[T, H * width]``."""
    return _mixer_backend(a).map_difference(a, gate, lam, factor, eps, width)


def output_gate(x, gate, width):
    """``x[T, H, pitch]``: the first ``width`` columns of every head times ``sigmoid(gate[T, H * width])``, ``[T, H * width]``."""
    return _mixer_backend(x).output_gate(x, gate, width)


def latent_layout(rank, rot, dtype, device):
    """``(column of the rotated part, width)`` of a cached latent row on ``device`` (see ``ops.cuda.latent_layout``)."""
    if torch.device(device).type == "cuda" and not _FORCE_TORCH:
        return native().latent_layout(rank, rot, dtype)
    return rank, rank + rot


def latent_store(proj, off_c, weight, eps, positions, cos_sin, slots, pages, q, off_rot, rank, rot, heads, dim, q_full=None,
                 queries=True, q_latent=None, width=None):
    """Latent attention's inputs from ``proj[T, *]`` (queries, ``dim`` plain and ``rot`` rotated dimensions per head, from
    column 0; ``rank`` latent columns and the shared key's ``rot`` columns from ``off_c``): the latent over its root mean
    square times ``weight``, and the shared key rotated (pairs ``2i, 2i + 1``), go to ``pages`` at the tokens' slots; the
    rotated dimensions of the queries go to ``q[T, H, *]`` from column ``off_rot``, zeros behind them, and whole queries (plain,
    rotated, zeros) to ``q_full[T, H, *]``; either may be ``None``.  ``pages`` ``None``: ``proj`` holds queries only (``width``: that
    of a page row).  ``queries=False``: it holds none, but with ``q_latent = (column, weight, out)`` another latent, which goes to
    ``out`` over its root mean square times ``weight``, zeros behind it."""
    _mixer_backend(proj).latent_store(proj, off_c, weight, eps, positions, cos_sin, slots, pages, q, off_rot, rank, rot, heads, dim,
                                      q_full, queries, q_latent, width)


def latent_attention(q, pages, rank, block_tables, cu_seqlens_q, kv_lens, scale, window=-1, max_q=None, max_kv=None, gate=None,
                     elsewhere=None, sink=None):
    """Causal attention of ``q[T, H, width]`` over the one key row per token in ``pages[blocks, block_size, 1, width]``, whose
    first ``rank`` columns are the value too; head outputs times ``sigmoid(gate[T, H])``.  ``[T, H, rank or more]``, zeros
    past ``rank``.  Sequences whose entry in ``elsewhere[B]`` is at least their number of tokens are left out (their rows are
    not written).  ``sink`` (fp32 ``[H]``): as in ``paged_attention``."""
    return _mixer_backend(q).latent_attention(q, pages, rank, block_tables, cu_seqlens_q, kv_lens, scale, window, max_q, max_kv,
                                              gate, elsewhere, sink)


def expanded_dims(dim, vdim, dtype, device):
    """Head widths of ``expanded_attention`` for ``dim`` query / key and ``vdim`` value dimensions, ``None``: not available."""
    if torch.device(device).type == "cuda" and not _FORCE_TORCH:
        return native().expanded_dims(dim, vdim, dtype)
    return None


def expanded_attention(q, kv, plan, cu_seqlens_q, scale, window, max_q, gate, out, sink=None):
    """Causal attention of ``q[T, H, dk]`` over keys and values written out for the step, ``kv[rows, H * dk + H * 128]``, laid out
    as ``plan`` (``models.mixers.Expansion``) says; rows of the plan's sequences are written to ``out[T, H, 128]``."""
    native().expanded_attention(q, kv, plan, cu_seqlens_q, scale, window, max_q, gate, out, sink)


def recurrent_pitch(dim, device):
    """Row pitch of a head's recurrent state (``dim`` key channels)."""
    if torch.device(device).type == "cuda" and not _FORCE_TORCH:
        return native().recurrent_pitch(dim)
    return dim


def conv_weights(parts, device):
    """Short convolutions ``[channels, taps]`` side by side as fp32 ``[rows, channels]``, oldest tap first; the kernels want
    a certain number of rows (absent taps are zero rows in front)."""
    w = torch.cat([p.float() for p in parts], dim=0).t()
    rows = native().conv_rows(w.shape[0]) if torch.device(device).type == "cuda" and not _FORCE_TORCH else w.shape[0]
    return torch.nn.functional.pad(w, (0, 0, rows - w.shape[0], 0)).contiguous().to(device)


def delta_inputs(proj, offs, a_pre, conv_t, a_log, dt_bias, cu, kv_lens, state_slots, conv_state, kv_heads, heads, dim, pitch,
                 vdim, single, head_decay=False):
    """Short convolutions (``conv_weights`` of q, k, v), unit norms, decays and write strengths of a gated delta rule;
    advances ``conv_state``.  Decays are one per head and key channel, or one per head (``head_decay``: ``a_pre`` and
    ``dt_bias`` have a value per head)."""
    return _mixer_backend(proj).delta_inputs(proj, offs, a_pre, conv_t, a_log, dt_bias, cu, kv_lens, state_slots, conv_state,
                                             kv_heads, heads, dim, pitch, vdim, single, head_decay)


def delta_scan(q, k, v, g, beta, qk, cu, kv_lens, state_slots, state, dim, max_q):
    """Gated delta rule over the step's tokens (decays ``g[T, H, pitch]`` or ``g[T, H]``); advances ``state`` and returns the
    read-outs, fp32 ``[T, H, vdim]``."""
    return _mixer_backend(v).delta_scan(q, k, v, g, beta, qk, cu, kv_lens, state_slots, state, dim, max_q)


def decay_scan(proj, offs, decay, cu, kv_lens, state_slots, state, heads, dim, vdim, max_q, act="silu", k_scale=1.0):
    """Linear attention with one decay per head on q, k, v (after ``act``: ``"silu"`` or ``""``), k times ``k_scale``; advances
    ``state``, fp32 ``[T, H, vdim]``."""
    return _mixer_backend(proj).decay_scan(proj, offs, decay, cu, kv_lens, state_slots, state, heads, dim, vdim, max_q, act, k_scale)


def gated_norm(o, gate, weight, eps, groups, out_cols, act="sigmoid"):
    """RMSNorm of ``o`` over each of ``groups`` equal parts, times ``weight``, times ``sigmoid(gate)`` or ``silu(gate)``;
    ``[T, out_cols]``."""
    return _mixer_backend(o).gated_norm(o, gate, weight, eps, groups, out_cols, act)


def _into(out, y):
    if out is None:
        return y
    if getattr(out, "is_peer_push", False):
        out = out.fallback      # no pushing kernel on this path: the reduction pulls from the plain buffer
    out.copy_(y.view_as(out))
    return out


def linear(x, weight, bias=None, out=None):
    """``x @ weight^T + bias``; ``out`` (bf16, contiguous) receives the result when given.  A weight with up to 7 more
    columns than ``x`` was padded at load to the 16-byte rows the GEMM fetches."""
    if 0 < weight.shape[1] - x.shape[-1] < 8:
        x = torch.nn.functional.pad(x, (0, weight.shape[1] - x.shape[-1]))
    if use_native(x) and x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16:
        return native().gemm_bf16(x, weight, bias, out=out)
    return _into(out, ref.linear(x, weight, bias))


def linear_shallow(x, weight):
    """Product over a short inner dimension (low-rank projections).  The persistent GEMM is built for deep K and its
    epilogue dominates here: 8192 x 4096 x 128 takes 77 us, the library's 19 us; few rows stay on the persistent one."""
    if use_native(x) and x.dtype == torch.bfloat16 and x.shape[0] >= 512 and weight.shape[1] <= 768:
        return torch.nn.functional.linear(x, weight)
    return linear(x, weight)


def fp8_quant_act(x, group=128):
    if use_native(x):
        return native().fp8_quant_act(x, group)
    return ref.fp8_quant_act(x, group)


def gemm_fp8_block(xq, xs, wq, ws, out_dtype=torch.bfloat16, bias=None, out=None):
    if use_native(xq):
        return native().gemm_fp8_block(xq, xs, wq, ws, out_dtype, bias, out=out)
    return _into(out, ref.gemm_fp8_block(xq, xs, wq, ws, out_dtype, bias))


def embedding(ids, table):
    if use_native(table):
        return native().embedding(ids, table)
    return ref.embedding(ids, table)


def argmax_logprob(logits):
    if use_native(logits):
        return native().argmax_logprob(logits)
    return ref.argmax_logprob(logits)


def has_fused_sample(scores) -> bool:
    return use_native(scores)


def fused_sample(scores, temperature=None, top_k=None, top_p=None, do_sample=None, seeds=None, steps=None, typical_p=None):
    """One-kernel temperature / top-k / top-p / typical-p / sampling on CUDA tensors (see ``ops.cuda.fused_sample``)."""
    return native().fused_sample(scores, temperature, top_k, top_p, do_sample, seeds, steps, typical_p=typical_p)


def penalties(scores, history, repetition_penalty=None, frequency_penalty=None):
    """fp32 copy of CUDA ``scores[B, V]`` with repetition / frequency penalties of ``history[B, L]`` applied."""
    return native().penalties(scores, history, repetition_penalty, frequency_penalty)


def moe_topk_softmax(router_logits, top_k, renormalize=True):
    if use_native(router_logits) and router_logits.shape[-1] <= 256 and top_k <= 8:
        return native().moe_topk_softmax(router_logits, top_k, renormalize)
    return ref.moe_topk_softmax(router_logits, top_k, renormalize)


def moe_sparsemixer(router_logits, jitter_eps=0.01):
    return ref.moe_sparsemixer(router_logits, jitter_eps)


def moe_experts(x, w_gate_up, w_down, topk_weights, topk_ids, act="silu", first: int = 0):
    """Routed experts ``first .. first + E_local - 1`` (``first`` > 0: an expert-parallel rank's share)."""
    if use_native(x) and x.dtype == torch.bfloat16 and w_gate_up.dtype == torch.bfloat16 and x.shape[1] % 8 == 0 \
            and (w_gate_up.shape[1] // 2) % 8 == 0 and w_gate_up.shape[0] <= 256 and topk_ids.shape[1] <= 8:
        return native().moe_experts(x, w_gate_up, w_down, topk_weights, topk_ids, act, first)
    return ref.moe_experts(x, w_gate_up, w_down, topk_weights, topk_ids, act, first)


# ---- routed experts of layers with an ``ExpertSpec`` ----------------------------------------------
def moe_route_sigmoid(x, weight, correction, top_k, scale):
    """Router product, sigmoid, corrected choice and weights in fp32: ``(weights [T, k], experts [T, k])``."""
    return _mixer_backend(x).moe_route_sigmoid(x, weight, correction, top_k, scale)


def moe_route_softmax(x, weight, bias, top_k):
    """Router product plus bias in fp32, the ``top_k`` largest logits and the softmax over them: ``(weights [T, k], experts
    [T, k])``."""
    return _mixer_backend(x).moe_route_softmax(x, weight, bias, top_k)


def plain_expert_weights(w_up, w_down, w_gate=None):
    """``[E, I, H]`` and ``[E, H, I]`` as the kernels want them: bf16 sizes brought to multiples of 8 with zeros.  With
    ``w_gate`` the first matrix is ``[E, 2 I, H]``, gate rows before up rows."""
    if use_native(w_up) and w_up.dtype == torch.bfloat16:
        pad = lambda w: None if w is None else torch.nn.functional.pad(w, (0, -w.shape[2] % 8, 0, -w.shape[1] % 8))
        w_up, w_down, w_gate = pad(w_up), pad(w_down), pad(w_gate)
    if w_gate is not None:
        w_up = torch.cat([w_gate, w_up], dim=1)
    return w_up.contiguous(), w_down.contiguous()


def moe_plain_experts(x, w_up, w_down, topk_weights, topk_ids, act, gated=False):
    """``sum over slots of weight * down(act(up x))``, or ``down(act(gate x) * up x)`` when ``gated`` (weights from
    ``plain_expert_weights``)."""
    return _mixer_backend(x).moe_plain_experts(x, w_up, w_down, topk_weights, topk_ids, act, gated)
