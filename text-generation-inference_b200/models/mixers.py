"""Token mixers of decoders whose layers differ, configured per layer by an ``arch.MixerSpec``.

Every mixer is called like ``decoder.Attention`` (``x, x_scale, meta, rotary, kv, reduce``), owns the tensors of its
cache (``cache_tensors``) and runs as a short sequence of fused ops:

    attention   qkv GEMM -> [short convolutions +] rotate + unit RMS + value mixing + page store -> paged attention
                -> o GEMM; or qkvg GEMM -> RMS of whole rows + temperature + page store -> paged attention -> output gate
                -> o GEMM; or, with two maps per head, qkvg GEMM -> page store -> paged attention -> difference of the maps
                + norm + gate -> o GEMM
    latent      GEMM for q, latent and gate (or for the queries' latent, then one for q) -> RMS of the latent, rotations,
                page store -> queries times the key
                up-projection -> attention over the latents (all heads read one row per token), gate -> value
                up-projection -> o GEMM; for sequences that bring many tokens -> keys and values of the visible tokens
                written out by one GEMM -> attention per head, gate -> o GEMM
    delta       one GEMM for q, k, v, write strengths and decay / gate inputs (-> low-rank decay / gate GEMMs)
                -> short convolutions + unit norms + decays -> state scan -> norm x gate -> o GEMM
    decay       one GEMM for q, k, v, gate -> state scan (SiLU applied on the way in, if any) -> norm x gate -> o GEMM

What a mixer reads may be convolved over time first (``InputConv``, part of the layer).
Recurrent layers keep, per slot of the state pool, the matrix state of every head (fp32, ``[H, vdim, pitch]``); layers
with short convolutions, attention layers included, the last ``taps - 1`` inputs of every channel.  Which tokens a
sequence brings and from which slot it continues is in the step's metadata, so prompts, portions of prompts and decoded
tokens are one code path.
"""
from __future__ import annotations

import math
import os
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from .. import ops
from ..utils.rotary import RotaryTable, scaled_frequencies, yarn_frequencies
from .arch import MixerSpec
from .layers import FastLinear, TensorParallelColumnLinear, TensorParallelRowLinear

ALIGN = 8       # elements: 16-byte rows and column offsets of bf16 operands


def _up(n: int) -> int:
    return (n + ALIGN - 1) // ALIGN * ALIGN


def pad_columns(w: torch.Tensor) -> torch.Tensor:
    """Weight ``[N, K]`` with K brought to a multiple of ``ALIGN`` (GEMM operands are fetched in 16-byte pieces)."""
    return torch.nn.functional.pad(w, (0, _up(w.shape[1]) - w.shape[1])).contiguous()


def _column_input(w: torch.Tensor) -> torch.Tensor:
    return pad_columns(w) if w.dtype == torch.bfloat16 else w.contiguous()


def stack_rows(parts: Sequence[torch.Tensor]) -> Tuple[torch.Tensor, List[int]]:
    """One matrix whose products are those of ``parts`` side by side; every part starts at a multiple of ``ALIGN``
    columns of the output (zero rows in between).  Returns ``(matrix, column offsets)``."""
    offs, rows = [], 0
    for p in parts:
        offs.append(rows)
        rows += _up(p.shape[0])
    w = parts[0].new_zeros(rows, parts[0].shape[1])
    for p, o in zip(parts, offs):
        w[o:o + p.shape[0]] = p
    return _column_input(w), offs


def spread_columns(w: torch.Tensor, heads: int, width: int, pitch: int) -> torch.Tensor:
    """Output projection ``[N, heads * width]`` for inputs whose heads are ``pitch`` columns apart."""
    if pitch == width:
        return _column_input(w)
    out = w.new_zeros(w.shape[0], heads, pitch)
    out[:, :, :width] = w.view(w.shape[0], heads, width)
    return out.view(w.shape[0], heads * pitch)


class RotaryTables:
    """Tables shared by the layers of a model that rotate alike."""

    def __init__(self, max_positions: int, device):
        self.max_positions, self.device = max_positions, device
        self._tables: Dict[tuple, RotaryTable] = {}

    def get(self, s: MixerSpec) -> RotaryTable:
        key = (s.rot_dims, s.rot_base, s.rot_scaling, s.rot_yarn)
        if key not in self._tables:
            freq, amp = (yarn_frequencies(s.rot_base, s.rot_dims, s.rot_yarn) if s.rot_yarn else
                         (scaled_frequencies(s.rot_base, s.rot_dims, s.rot_scaling), 1.0))
            self._tables[key] = RotaryTable.from_frequencies(freq, self.max_positions, amplitude=amp).to(self.device)
        return self._tables[key]


class Mixer:
    def __init__(self, spec: MixerSpec, prefix: str, weights, idx: int, eps: float, comm=None):
        self.spec, self.prefix, self.weights, self.layer_idx, self.eps, self.comm = spec, prefix, weights, idx, eps, comm
        self.dtype, self.device, self.pg = weights.dtype, weights.device, weights.process_group

    def tensor(self, name: str) -> torch.Tensor:
        return self.weights.get_tensor(f"{self.prefix}.{name}")

    def f32(self, name: str) -> torch.Tensor:
        return self.weights.get_tensor(f"{self.prefix}.{name}", to_dtype=False).float().contiguous()

    def fused(self, names: Sequence[str], bias: bool = False) -> Tuple[TensorParallelColumnLinear, List[int]]:
        w, offs = stack_rows([self.tensor(n) for n in names])
        b = None
        if bias:
            b = w.new_zeros(w.shape[0])
            for n, o in zip(names, offs):
                part = self.tensor(f"{n}.b")
                b[o:o + part.shape[0]] = part
        return TensorParallelColumnLinear(FastLinear(w, b)), offs

    def load_conv(self) -> None:
        """Convolution weights of q, k and v side by side (channels of q first)."""
        parts = [self.f32(f"{n}.conv") for n in ("q", "k", "v")]
        self.channels, self.taps = sum(p.shape[0] for p in parts), parts[0].shape[1]
        self.conv = ops.conv_weights(parts, self.device)

    def conv_state(self, slots: int, device) -> torch.Tensor:
        """Last ``taps - 1`` inputs of every channel, oldest first, per slot."""
        return torch.zeros(slots, self.taps - 1, self.channels, dtype=self.dtype, device=device)

    def row(self, w: torch.Tensor) -> TensorParallelRowLinear:
        return TensorParallelRowLinear(FastLinear(w), self.pg, self.comm)

    input_conv: Optional["InputConv"] = None        # of the layer, which applies it; its state is kept with the mixer's

    def page_tensors(self, num_blocks: int, block_size: int, device) -> Tuple[torch.Tensor, ...]:
        return ()

    def state_tensors(self, slots: int, device) -> Tuple[torch.Tensor, ...]:
        return ()

    def cache_tensors(self, num_blocks: int, block_size: int, slots: int, device) -> Tuple[torch.Tensor, ...]:
        """What the mixer keeps between steps: pages (addressed by token), then states (addressed by request)."""
        return self.page_tensors(num_blocks, block_size, device) + self.slot_tensors(slots, device)

    def slot_tensors(self, slots: int, device) -> Tuple[torch.Tensor, ...]:
        """The mixer's states and, last, that of the input convolution."""
        conv = () if self.input_conv is None else (self.input_conv.state(slots, device),)
        return self.state_tensors(slots, device) + conv

    def state_bytes(self) -> int:
        """Bytes of one slot of the state pool."""
        return sum(t.numel() * t.element_size() for t in self.slot_tensors(1, "meta"))

    def page_bytes(self, block_size: int) -> int:
        return sum(t.numel() * t.element_size() for t in self.page_tensors(1, block_size, "meta"))


class InputConv:
    """``h + conv(h)``: a causal convolution over time on every channel of what a mixer reads."""

    def __init__(self, weight: torch.Tensor, dtype, device):
        self.channels, self.taps = weight.shape
        w = weight.float().t().contiguous().to(device)        # [taps, channels], oldest input first
        w[-1] += 1                                             # the input itself
        self.weight, self.dtype = w, dtype

    def state(self, slots: int, device) -> torch.Tensor:
        return torch.zeros(slots, self.taps - 1, self.channels, dtype=self.dtype, device=device)

    def at(self, meta, state: torch.Tensor) -> "ops.ShortConv":
        return ops.ShortConv(self.weight, state, meta.cu_seqlens_q, meta.kv_lens, meta.state_slots, meta.max_q == 1)


class MixedAttention(Mixer):
    """Paged attention with its own head sizes: short convolutions of q, k and v, rotation of the first dimensions,
    weightless RMS of q and k after it, values mixed with an earlier layer's, keys limited to the query's chunk or window,
    a sink in the softmax.  Or, without any of the first four: weighted RMS of q and k over all heads, queries times a factor
    of their position, keys and values of an earlier layer.  Capped scores and an output gate go with either.  Or, without
    any of these but the gate: two maps per head over the same values, and their normed difference.  Both maps of a key lie
    side by side in one page row, and a query map is a query of its own with zeros at the other map's place."""

    def __init__(self, spec, prefix, weights, idx, eps, comm=None, rotary: Optional[RotaryTables] = None):
        super().__init__(spec, prefix, weights, idx, eps, comm)
        s = spec
        if s.row_norm and (s.short_conv or s.rot_dims or s.qk_unit_rms or s.v_mix):
            raise NotImplementedError(f"{prefix}: a norm over whole rows beside convolutions, rotation, unit norms or value mixing")
        self.maps = 1 if s.diff is None else 2
        if s.diff is not None and (s.row_norm or s.short_conv or s.rot_dims or s.qk_unit_rms or s.v_mix or s.softcap or s.sink
                                   or s.learned_sink or s.kv_from is not None or s.out_gate not in ("", "head")):
            raise NotImplementedError(f"{prefix}: differences of two maps beside norms, rotation, sinks or shared keys")
        if s.diff is None and s.out_gate not in ("", "element"):
            raise NotImplementedError(f"{prefix}: output gate {s.out_gate!r} on attention of one map")
        own = ["q", "k", "v"] if s.kv_from is None else ["q"]
        self.qkv, offs = self.fused(own + (["g"] if s.out_gate else []), bias=s.qkv_bias)
        self.offs, self.off_gate = offs[:len(own)], offs[-1]
        self.q_norm, self.k_norm = (self.f32(f"{n}.norm") if s.row_norm and n in own else None for n in ("q", "k"))
        self.sink = self.f32("sink") if s.learned_sink else (True if s.sink else None)
        self.conv = None
        if s.short_conv:
            self.load_conv()
        self.v_lambda = float(self.f32("vmix").reshape(-1)[0]) if s.v_mix and weights.has_tensor(f"{prefix}.vmix") else 0.0
        if s.diff is not None:
            part = lambda i: math.exp(float((self.f32(f"lq{i}").double() * self.f32(f"lk{i}").double()).sum()))
            self.map_lambda = part(1) - part(2) + s.diff
        self.kd, self.vd = ops.attention_pitch(self.maps * s.dim, s.vdim, self.dtype, self.device)
        # a gate (or the difference of maps) packs the heads again
        self.o = self.row(_column_input(self.tensor("o")) if s.out_gate or s.diff is not None else
                          spread_columns(self.tensor("o"), s.heads, s.vdim, self.vd))
        self.rotary = rotary.get(s)

    def page_tensors(self, num_blocks: int, block_size: int, device):
        if self.spec.kv_from is not None:
            return ()
        # zeros: the kernels never write the padding columns of a page, and padded queries must meet zeros there
        return tuple(torch.zeros(num_blocks, block_size, self.spec.kv_heads, d, dtype=self.dtype, device=device)
                     for d in (self.kd, self.vd))

    def state_tensors(self, slots: int, device):
        return () if self.conv is None else (self.conv_state(slots, device),)

    def __call__(self, x, x_scale, meta, rotary, kv, reduce: bool = True, out=None):
        s = self.spec
        k_cache, v_cache = kv[:2]
        proj = self.qkv(x)
        if s.row_norm:
            q = ops.row_norm_store(proj, self.offs, meta.positions, meta.slots, k_cache, v_cache, self.q_norm, self.k_norm, self.eps,
                                   s.heads, s.kv_heads, s.dim, s.vdim, self.kd, s.q_temp)
        elif s.diff is not None:
            q = ops.map_store(proj, self.offs, meta.slots, k_cache, v_cache, s.heads, s.kv_heads, s.dim, s.vdim)
        else:
            q = self._rotated(proj, meta, kv)
        a = ops.paged_attention(q, k_cache, v_cache, meta.block_tables, meta.cu_seqlens_q, meta.kv_lens, s.scale,
                                window=s.window or -1, softcap=s.softcap, max_q=meta.max_q, max_kv=meta.max_kv, chunk=s.chunk,
                                sink=self.sink, keep=s.keep_first)
        if s.diff is not None:
            gate = proj[:, self.off_gate:self.off_gate + s.heads] if s.out_gate else None
            a = ops.map_difference(a, gate, self.map_lambda, 1.0 - s.diff, self.eps, s.vdim)
        elif s.out_gate:
            a = ops.output_gate(a, proj[:, self.off_gate:self.off_gate + s.heads * s.vdim], s.vdim)
        return self.o(a.view(a.shape[0], -1), reduce=reduce, out=out)

    def _rotated(self, proj, meta, kv):
        s = self.spec
        k_cache, v_cache = kv[:2]
        v_first = None
        if s.v_mix:
            v_first = meta.v_first
            if v_first is None:      # the first such layer: its values are what the later ones mix in
                meta.v_first = proj[:, self.offs[2]:self.offs[2] + s.kv_heads * s.vdim]
        conv = None
        if self.conv is not None:
            conv = ops.ShortConv(self.conv, kv[2], meta.cu_seqlens_q, meta.kv_lens, meta.state_slots, meta.max_q == 1)
        return ops.rotate_norm_store(proj, self.offs, meta.positions, self.rotary.cos_sin, meta.slots, k_cache, v_cache, s.heads,
                                     s.kv_heads, s.dim, s.vdim, s.rot_dims, s.qk_unit_rms, self.eps, v_first, self.v_lambda,
                                     s.rot_interleaved, conv)


# tokens of a sequence in one step from which its latents are expanded to keys and values per head, and the most rows
# that a step expands (their keys and values are held for one layer at a time)
EXPAND_TOKENS = int(os.environ.get("TGI_B200_LATENT_EXPAND", "64"))
EXPAND_ROWS = int(os.environ.get("TGI_B200_LATENT_EXPAND_ROWS", "131072"))
EXPAND_GROUP = 16           # rows of a group that a table entry names


@dataclass
class Expansion:
    """Tokens whose keys and values a step writes out, for layers with one window: for every expanded sequence those its
    queries see, from a multiple of ``EXPAND_GROUP`` positions on.  Positions count from there (scores do not depend on it)."""

    rows: torch.Tensor          # [R] page row (slot) of every expanded token; gaps at the sequences' ends repeat one
    tables: torch.Tensor        # [B, *] groups of rows of a sequence
    kv_lens: torch.Tensor       # [B] expanded tokens, 0: the sequence is not expanded
    queries: torch.Tensor       # rows of the step that belong to expanded sequences
    all: bool                   # every sequence that brings tokens is expanded
    rest_max_q: int             # most tokens of the others


def plan_expansion(window: int, starts: Sequence[int], counts: Sequence[int], slots: Sequence[np.ndarray]):
    """Host arrays of an ``Expansion`` (``rows, tables, kv_lens, queries``) with its two scalars, or ``None``.  ``starts``:
    position of a sequence's first token of the step, ``slots``: page rows of its positions."""
    g, total, at, rest = EXPAND_GROUP, 0, 0, 0
    rows, groups, queries = [], [], []
    kv = np.zeros(len(counts), dtype=np.int32)
    for b, (s, n) in enumerate(zip(starts, counts)):
        first = max(0, s - window + 1) // g * g if window > 0 else 0
        length = s + n - first
        padded = -(-length // g) * g
        if n >= EXPAND_TOKENS and total + padded <= EXPAND_ROWS:
            own = np.zeros(padded, dtype=np.int32)
            own[:length] = slots[b][first:s + n]
            own[length:] = own[0]
            rows.append(own)
            groups.append(np.arange(total // g, (total + padded) // g, dtype=np.int32))
            queries.append(np.arange(at, at + n, dtype=np.int32))
            kv[b] = length
            total += padded
        else:
            groups.append(np.zeros(0, dtype=np.int32))
            rest = max(rest, n)
        at += n
    if not rows:
        return None
    tables = np.zeros((len(counts), max(len(x) for x in groups)), dtype=np.int32)
    for b, x in enumerate(groups):
        tables[b, :len(x)] = x
    return (np.concatenate(rows), tables, kv, np.concatenate(queries)), (rest == 0, rest)


class LatentAttention(Mixer):
    """Attention whose keys and values are up-projections of one latent per token, beside which a rotated key part that all
    heads share may stand.  Only latent and rotated part are cached.  The up-projections are moved to the other side of the
    attention: ``q . (W_uk c) = (W_uk^T q) . c`` and ``sum p W_uv c = W_uv sum p c``, so every head attends to the same rows.
    That costs more operations per query and key, so sequences that bring many tokens attend to keys and values written out
    (``Expansion``), one matrix product of the cached rows (the rotated part passes through a block of ones)."""

    def __init__(self, spec, prefix, weights, idx, eps, comm=None, rotary: Optional[RotaryTables] = None):
        super().__init__(spec, prefix, weights, idx, eps, comm)
        s = spec
        # rotations pair neighbours: with halves for pairs, the rows of the projections are brought to that order
        self.order = None if s.rot_interleaved or not s.rot_dims else torch.arange(s.rot_dims).view(2, -1).t().reshape(-1)
        names = ["dq" if s.q_rank else "q", "dkv"] + (["g"] if s.out_gate else [])
        w, self.offs = stack_rows([self._rows(n) for n in names])
        self.proj = TensorParallelColumnLinear(FastLinear(w))
        self.norm = self.f32("dkv.norm")
        if s.q_rank:
            self.q_norm = self.f32("dq.norm")
            self.uq = TensorParallelColumnLinear(FastLinear(stack_rows([self._rows("uq")])[0]))
            self.q_cols = self.uq.linear.weight.shape[1]
        self.sink = self.f32("sink") if s.learned_sink else None
        self.off_rot, self.width = ops.latent_layout(s.kv_rank, s.rot_dims, self.dtype, self.device)
        pad = (0, self.off_rot - s.kv_rank)
        self.uk, self.uv = (torch.nn.functional.pad(self.tensor(n).view(s.heads, d, s.kv_rank), pad).contiguous()
                            for n, d in (("uk", s.dim), ("uv", s.vdim)))         # [H, d, columns of the latent]
        self.full = ops.expanded_dims(s.dim + s.rot_dims, s.vdim, self.dtype, self.device)
        if self.full is not None:
            dk, dv = self.full
            k, v = self.uk.new_zeros(s.heads, dk, self.width), self.uv.new_zeros(s.heads, dv, self.width)
            k[:, :s.dim, :self.off_rot], v[:, :s.vdim, :self.off_rot] = self.uk, self.uv
            turn = torch.arange(s.rot_dims, device=self.device)
            k[:, s.dim + turn, self.off_rot + turn] = 1
            self.expand = torch.cat([k.view(-1, self.width), v.view(-1, self.width)])
        self.o = self.row(_column_input(self.tensor("o")))
        self.rotary = rotary.get(s)

    def _rows(self, name: str) -> torch.Tensor:
        s, w = self.spec, self.tensor(name)
        if self.order is not None and name == "dkv":
            w = torch.cat([w[:s.kv_rank], w[s.kv_rank:][self.order.to(w.device)]])
        elif self.order is not None and name in ("q", "uq"):
            rows = torch.cat([torch.arange(s.dim), s.dim + self.order]).to(w.device)
            w = w.view(s.heads, s.dim + s.rot_dims, -1)[:, rows].reshape(w.shape)
        return w

    def page_tensors(self, num_blocks: int, block_size: int, device):
        # zeros: the kernels never write the padding columns
        return (torch.zeros(num_blocks, block_size, 1, self.width, dtype=self.dtype, device=device),)

    def __call__(self, x, x_scale, meta, rotary, kv, reduce: bool = True, out=None):
        s, T = self.spec, x.shape[0]
        pages, = kv
        proj = self.proj(x)
        plan = meta.expansions.get(s.window) if meta.expansions and self.full is not None else None
        rest = plan is None or not plan.all
        q = proj.new_empty(T, s.heads, self.width) if rest else None
        q_full = None if plan is None else proj.new_empty(T, s.heads, self.full[0])
        places = (self.off_rot, s.kv_rank, s.rot_dims, s.heads, s.dim)
        turns = (meta.positions, self.rotary.cos_sin, meta.slots)
        if s.q_rank:
            cq = proj.new_empty(T, self.q_cols)
            ops.latent_store(proj, self.offs[1], self.norm, self.eps, *turns, pages, None, *places, queries=False,
                             q_latent=(self.offs[0], self.q_norm, cq))
            queries = self.uq(cq)
            ops.latent_store(queries, 0, None, self.eps, *turns, None, q, *places, q_full, width=self.width)
        else:
            queries = proj
            ops.latent_store(proj, self.offs[1], self.norm, self.eps, *turns, pages, q, *places, q_full)
        gate = proj[:, self.offs[2]:self.offs[2] + s.heads] if s.out_gate == "head" else None
        y = proj.new_empty(T, s.heads, s.vdim)
        if rest:
            plain = queries[:, :s.heads * (s.dim + s.rot_dims)].unflatten(1, (s.heads, -1))[..., :s.dim]
            torch.bmm(plain.transpose(0, 1), self.uk, out=q[..., :self.off_rot].transpose(0, 1))
            a = ops.latent_attention(q, pages, s.kv_rank, meta.block_tables, meta.cu_seqlens_q, meta.kv_lens, s.scale,
                                     s.window or -1, meta.max_q if plan is None else plan.rest_max_q, meta.max_kv, gate,
                                     None if plan is None else plan.kv_lens, self.sink)
            torch.bmm(a.transpose(0, 1), self.uv[..., :a.shape[2]].transpose(1, 2), out=y.transpose(0, 1))
        if plan is not None:
            written = ops.linear_shallow(pages.view(-1, self.width).index_select(0, plan.rows), self.expand)
            o = y if s.vdim == self.full[1] else proj.new_empty(T, s.heads, self.full[1])
            ops.expanded_attention(q_full, written, plan, meta.cu_seqlens_q, s.scale, s.window or -1, meta.max_q, gate, o, self.sink)
            if o is not y and plan.all and s.out_gate == "element":
                y = o                    # the gate packs the heads
            elif o is not y:
                y.index_copy_(0, plan.queries.long(), o.index_select(0, plan.queries)[..., :s.vdim])
        if s.out_gate == "element":
            y = ops.output_gate(y, proj[:, self.offs[2]:self.offs[2] + s.heads * s.vdim], s.vdim)
        return self.o(y.view(T, -1), reduce=reduce, out=out)


class GatedDelta(Mixer):
    """Gated delta rule whose decay acts per head and key channel (decay and gate of low rank) or per head."""

    def __init__(self, spec, prefix, weights, idx, eps, comm=None, rotary=None):
        super().__init__(spec, prefix, weights, idx, eps, comm)
        s = spec
        # decay and gate: read where the fused product leaves them, or low-rank products of what it leaves there
        self.proj, self.offs = self.fused(["q", "k", "v", "b"] + (["a", "g"] if s.head_decay else ["a1", "g1"]))
        self.load_conv()
        if not s.head_decay:
            self.a_rank, self.g_rank = (_up(self.weights.get_shape(f"{prefix}.{n}")[0]) for n in ("a1", "g1"))
            # K padded like the rows of a1 / g1: their outputs are read where the fused product left them
            self.a2, self.g2 = (pad_columns(self.tensor(n)) for n in ("a2", "g2"))
        self.a_log, self.dt_bias, self.norm = self.f32("A_log"), self.f32("dt_bias"), self.f32("norm")
        self.pitch = ops.recurrent_pitch(s.dim, self.device)
        self.o = self.row(_column_input(self.tensor("o")))
        self.out_cols = self.o.linear.weight.shape[1]

    def state_tensors(self, slots: int, device):
        s = self.spec
        return (self.conv_state(slots, device),
                torch.zeros(slots, s.heads, s.vdim, self.pitch, dtype=torch.float32, device=device))

    def __call__(self, x, x_scale, meta, rotary, kv, reduce: bool = True, out=None):
        s = self.spec
        conv_state, state = kv
        p = self.proj(x)
        if s.head_decay:
            a, g = (p[:, o:o + n] for o, n in zip(self.offs[4:], (s.heads, s.heads * s.vdim)))
        else:
            a = ops.linear_shallow(p[:, self.offs[4]:self.offs[4] + self.a_rank], self.a2)
            g = ops.linear_shallow(p[:, self.offs[5]:self.offs[5] + self.g_rank], self.g2)
        q, k, v, decay, beta, qk = ops.delta_inputs(
            p, self.offs, a, self.conv, self.a_log, self.dt_bias, meta.cu_seqlens_q, meta.kv_lens, meta.state_slots,
            conv_state, s.kv_heads, s.heads, s.dim, self.pitch, s.vdim, meta.max_q == 1, s.head_decay)
        o = ops.delta_scan(q, k, v, decay, beta, qk, meta.cu_seqlens_q, meta.kv_lens, meta.state_slots, state, s.dim, meta.max_q)
        y = ops.gated_norm(o, g, self.norm, self.eps, s.heads, self.out_cols, s.gate_act)
        return self.o(y, reduce=reduce, out=out)


class DecayAttention(Mixer):
    """Linear attention whose state shrinks by a fixed factor per head and token."""

    def __init__(self, spec, prefix, weights, idx, eps, comm=None, rotary=None):
        super().__init__(spec, prefix, weights, idx, eps, comm)
        s = spec
        if len(s.decay) != s.heads:
            raise ValueError(f"{prefix}: {len(s.decay)} decays for {s.heads} heads")
        self.proj, self.offs = self.fused(["q", "k", "v", "g"])
        self.decay = torch.tensor(s.decay, dtype=torch.float32, device=self.device)
        self.groups = s.heads if s.head_norm else 1
        self.norm = torch.ones(s.vdim, dtype=torch.float32, device=self.device) if s.head_norm else self.f32("norm")
        self.pitch = ops.recurrent_pitch(s.dim, self.device)
        self.o = self.row(_column_input(self.tensor("o")))
        self.out_cols = self.o.linear.weight.shape[1]

    def state_tensors(self, slots: int, device):
        s = self.spec
        return (torch.zeros(slots, s.heads, s.vdim, self.pitch, dtype=torch.float32, device=device),)

    def __call__(self, x, x_scale, meta, rotary, kv, reduce: bool = True, out=None):
        s = self.spec
        p = self.proj(x)
        o = ops.decay_scan(p, self.offs, self.decay, meta.cu_seqlens_q, meta.kv_lens, meta.state_slots, kv[0], s.heads, s.dim,
                           s.vdim, meta.max_q, s.qkv_act, s.k_scale)
        y = ops.gated_norm(o, p[:, self.offs[3]:], self.norm, self.eps, self.groups, self.out_cols, s.gate_act)
        return self.o(y, reduce=reduce, out=out)


MIXERS = {"attention": MixedAttention, "latent": LatentAttention, "delta": GatedDelta, "decay": DecayAttention}


def load_mixer(spec: MixerSpec, prefix: str, weights, idx: int, eps: float, comm, rotary: RotaryTables,
               input_conv: Optional[str] = None) -> Mixer:
    """``input_conv``: tensor of the layer's input convolution."""
    mixer = MIXERS[spec.kind](spec, prefix, weights, idx, eps, comm, rotary)
    if spec.input_conv:
        w = weights.get_tensor(input_conv, to_dtype=False)
        if w.shape[1] != spec.input_conv:
            raise ValueError(f"{input_conv}: {w.shape[1]} taps instead of {spec.input_conv}")
        mixer.input_conv = InputConv(w, weights.dtype, weights.device)
    return mixer
