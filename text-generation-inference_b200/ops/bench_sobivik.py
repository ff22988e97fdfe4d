"""Shapes and kernels of ``python bench.py --model sobivik-bf16`` (see ``bench_hybrid``): a Sobivik decoder beside a Fuzuvik
shape of the same width, depth, heads and parameters whose layers are linear attention and attention in the same order."""
from __future__ import annotations

import math

import torch


def sobivik_like(width: int, layers: int, vocab: int, window: int) -> dict:
    """Heads of 128 (two maps of 64 in differential attention, 128 + 64 rotated in latent attention), latents of 512."""
    from ..utils import synthetic as syn

    h, dense = width // 128, syn.kipedra_dense((8 * width // 3 + 127) // 128 * 128)
    ret = syn.sobivik_retention(h, 128, 128, mlp=dense)
    kinds = [ret, syn.sobivik_latent(h, 128, 128, 3 * width // 8, 512, 64, window, 500000.0, (8.0, 32.0, 1.0, 4096), mlp=dense),
             syn.sobivik_attention(h, h // 4, 64, 128, window, 4, 0.5, mlp=dense), ret]
    return syn.sobivik_config([kinds[i % 4] for i in range(layers)], width=width, vocab=vocab, eps=1e-6)


def fuzuvik_relative(width: int, layers: int, vocab: int, window: int) -> dict:
    """Linear attention, attention, attention, linear attention; chunks as long as the windows."""
    from .bench_hybrid import fuzuvik_like

    cfg = fuzuvik_like(width, 4, vocab, window)
    attn, linear = cfg["layers"][0], cfg["layers"][3]
    cfg["layers"] = [(linear, attn, attn, linear)[i % 4] for i in range(layers)]
    return cfg


def sobivik_rows(dev, width: int, window: int, prefill, decode) -> list:
    """Every kernel of the design at layer size, and the like kernels of the Fuzuvik, Kipedra, Gisilix and Llama shapes."""
    import numpy as np

    from .. import ops
    from . import cuda as K
    from ..models.arch import MixerSpec
    from ..models.mixers import Expansion, RotaryTables, plan_expansion
    from .bench_hybrid import KernelTimer

    H, G, d, rank, rot, qr, taps, index = width // 128, width // 512, 128, 512, 64, 3 * width // 8, 4, 4
    kt = KernelTimer(dev)
    bf, f32 = torch.bfloat16, torch.float32
    tab = RotaryTables(16384, dev).get(MixerSpec("latent", H, 1, d, d, rot_dims=rot, rot_base=500000.0)).cos_sin
    full_tab = RotaryTables(16384, dev).get(MixerSpec("attention", H, G, d, d, rot_dims=d, rot_base=500000.0)).cos_sin
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rn = lambda *s, dt=bf, std=1.0: (torch.randn(*s, device=dev, dtype=f32) * std).to(dt)
    gemm = lambda t, n, k: ((t + n) * k * 2 + t * n * 2, 2.0 * t * n * k)
    for label, B, n, ctx in [("prefill", *prefill, prefill[1]), ("decode", decode[0], 1, decode[1])]:
        T, one = B * n, n == 1
        tag = f"{label} {B}x{n}" + (f" @{ctx}" if one else "")
        cu, kv, slots = i32([i * n for i in range(B + 1)]), i32([ctx] * B), i32(list(range(B)))
        per = math.ceil(ctx / 16)
        bt = torch.arange(B * per, dtype=torch.int32, device=dev).view(B, per)
        pos = i32([ctx - n + i for _ in range(B) for i in range(n)])
        page = i32([b * per * 16 + ctx - n + i for b in range(B) for i in range(n)])
        pairs = lambda w: B * sum(min(i + 1, w) if w else i + 1 for i in range(ctx - n, ctx))
        seen = lambda w: B * min(ctx, w + n - 1 if w else ctx)
        # ---- stream: the step between mixer and feed-forward, and that between layers, the fifth result in
        res, dl, x, w = rn(T, width, dt=f32), rn(T, width), rn(T, width), rn(width)
        streams, avg = rn(index + 1, T, width, dt=f32), torch.full((index + 1,), 0.2, device=dev)
        cw, past = rn(taps, width, dt=f32), torch.zeros(B, taps - 1, width, dtype=bf, device=dev)
        conv = ops.ShortConv(cw, past, cu, kv, slots, one)
        kt(f"{tag}: norm + residual (fp32) + norm", lambda: ops.stream_step(dl, w, res, w, 1e-6), T * width * 12)
        cb = B * (taps - 1) * width * 2
        if one:
            kt(f"{tag}: norm + residual + sum of 5 results + norm + convolution", lambda: ops.stream_step(
                dl, w, res, w, 1e-6, average=avg, streams=streams, conv=conv), T * width * (16 + 4 * index) + 2 * cb)
        else:
            kt(f"{tag}: norm + residual + sum of 5 results + norm", lambda: ops.stream_step(
                dl, w, res, w, 1e-6, average=avg, streams=streams), T * width * (16 + 4 * index))
            kt(f"{tag}: input convolution", lambda: K.input_conv(x, conv), T * width * 4 + cb)
        kt(f"{tag}: [fuzuvik] residual (fp32) + norm", lambda: ops.residual_norm(dl, res, w, 1e-6), T * width * 12)
        del streams
        # ---- retention
        y, dec, S = rn(T, 4 * H * d), torch.full((H,), 0.99, device=dev), torch.zeros(B, H, d, d, device=dev)
        offs = [0, H * d, 2 * H * d]
        st = B * H * d * d * 4 * (2 if one else 1)
        for name, kw in (("retention scan", dict(act="", k_scale=d ** -0.5)), ("[fuzuvik] decay scan", {})):
            kt(f"{tag}: {name}", lambda: ops.decay_scan(y, offs, dec, cu, kv, slots, S, H, d, d, n, **kw),
               T * H * d * (3 * 2 + 4) + st, 5.0 * T * H * d * d, "fp32")
        o, ones, whole = rn(T, H, d, dt=f32), torch.ones(d, device=dev), torch.ones(H * d, device=dev)
        kt(f"{tag}: norm x silu gate, per head", lambda: ops.gated_norm(o, y[:, 3 * H * d:], ones, 1e-6, H, H * d, "silu"), T * H * d * 8)
        kt(f"{tag}: [fuzuvik] norm x gate, whole row", lambda: ops.gated_norm(o, y[:, 3 * H * d:], whole, 1e-6, 1, H * d), T * H * d * 8)
        wg = rn(4 * H * d, width)
        kt(f"{tag}: GEMM q k v g", lambda: ops.linear(x, wg), *gemm(T, 4 * H * d, width))
        del S, o, y, wg
        # ---- differential attention
        qw = (H + 2 * G) * d
        hp = (H + 7) // 8 * 8
        proj, offs = rn(T, qw + hp), [0, H * d, (H + G) * d]
        kc, vc = rn(B * per, 16, G, d), rn(B * per, 16, G, d)
        kt(f"{tag}: queries of both maps + store", lambda: ops.map_store(proj, offs, page, kc, vc, H, G, d // 2, d),
           T * (H + 2 * G + 2 * H + 2 * G) * d * 2)
        plain = proj[:, :qw].contiguous()
        kt(f"{tag}: [llama] rope + store", lambda: ops.rope_and_cache(plain, pos, full_tab, page, kc, vc, H, G, d, d), T * qw * 4)
        q2 = ops.map_store(proj, offs, page, kc, vc, H, G, d // 2, d)
        q1 = q2[:, :H].contiguous()
        for name, q, heads, keep, flops in (("attention of two maps, window + kept tokens", q2, 2 * H, 4, 2 * (d // 2 + d)),
                                            ("[kipedra] attention, window", q1, H, 0, 4 * d)):
            kt(f"{tag}: {name}", lambda: ops.paged_attention(q, kc, vc, bt, cu, kv, 0.1, window=window, max_q=n, max_kv=ctx, keep=keep),
               (seen(window) * 2 * G + 2 * T * heads) * d * 2, 0.0 if one else float(flops) * pairs(window) * heads)
        a = rn(T, 2 * H, d)
        kt(f"{tag}: difference of maps + norm + gate", lambda: ops.map_difference(a, proj[:, qw:qw + H], 0.4, 0.5, 1e-6, d), T * H * d * 6)
        kt(f"{tag}: [gisilix] output gate", lambda: ops.output_gate(q1, proj[:, :H * d], d), T * H * d * 6)
        wq = rn(qw + hp, width)
        kt(f"{tag}: GEMM q k v g (maps)", lambda: ops.linear(x, wq), *gemm(T, qw + hp, width))
        del kc, vc, a, q1, q2, wq, plain
        # ---- latent attention
        cols = qr + rank + rot + H * d
        off, wide = ops.latent_layout(rank, rot, bf, dev)
        proj, pages, norm, qnorm = rn(T, cols), rn(B * per, 16, 1, wide), torch.ones(rank, device=dev), torch.ones(qr, device=dev)
        sink, gate = torch.zeros(H, device=dev), rn(T, H)
        wl, wu = rn(cols, width), rn(H * (d + rot), qr)
        kt(f"{tag}: GEMM dq dkv g", lambda: ops.linear(x, wl), *gemm(T, cols, width))
        cq = torch.empty(T, qr, dtype=bf, device=dev)
        kt(f"{tag}: latent norms + rotation + store", lambda: ops.latent_store(
            proj, qr, norm, 1e-6, pos, tab, page, pages, None, off, rank, rot, H, d, queries=False, q_latent=(0, qnorm, cq)),
           T * (qr + rank + rot) * 4)
        kt(f"{tag}: GEMM uq", lambda: ops.linear(cq, wu), *gemm(T, H * (d + rot), qr))
        qp = rn(T, H * (d + rot))
        mine, theirs = dict(sink=sink), dict(gate=gate)
        if one:
            lq = rn(T, H, wide)
            kt(f"{tag}: rotation of queries", lambda: ops.latent_store(qp, 0, None, 1e-6, pos, tab, page, None, lq, off, rank, rot, H, d, width=wide),
               T * H * rot * 4)
            uk, uv = rn(H, d, rank), rn(H, d, rank)
            heads = qp.view(T, H, -1)[..., :d]
            kt(f"{tag}: queries x key up-projection", lambda: torch.bmm(heads.transpose(0, 1), uk, out=lq[..., :off].transpose(0, 1)),
               H * d * rank * 2 + T * H * (d + rank) * 2, 2.0 * T * H * d * rank)
            for name, kw in (("latent attention, window + sinks", mine), ("[gisilix] latent attention, window + gate", theirs)):
                a = ops.latent_attention(lq, pages, rank, bt, cu, kv, 0.07, window, 1, ctx, **kw)
                kt(f"{tag}: {name}", lambda: ops.latent_attention(lq, pages, rank, bt, cu, kv, 0.07, window, 1, ctx, **kw),
                   seen(window) * wide * 2 + T * H * (wide + rank) * 2, 2.0 * pairs(window) * H * (wide + rank))
            yv = torch.empty(T, H, d, dtype=bf, device=dev)
            kt(f"{tag}: outputs x value up-projection", lambda: torch.bmm(a.transpose(0, 1), uv.transpose(1, 2), out=yv.transpose(0, 1)),
               H * d * rank * 2 + T * H * (d + rank) * 2, 2.0 * T * H * d * rank)
        else:
            fq, yv = rn(T, H, 192), torch.empty(T, H, d, dtype=bf, device=dev)
            kt(f"{tag}: rotation of queries", lambda: ops.latent_store(qp, 0, None, 1e-6, pos, tab, page, None, None, off, rank, rot, H, d, fq, width=wide),
               T * H * (d + rot) * 4)
            arrays, scalars = plan_expansion(window, [0] * B, [n] * B, [np.arange(b * per * 16, (b + 1) * per * 16, dtype=np.int32) for b in range(B)])
            plan = Expansion(*(torch.from_numpy(z).to(dev) for z in arrays), *scalars)
            R, ew = plan.rows.numel(), rn(H * 320, wide, std=0.05)
            rows = pages.view(-1, wide).index_select(0, plan.rows)
            kt(f"{tag}: gather of latent rows", lambda: pages.view(-1, wide).index_select(0, plan.rows), R * wide * 4)
            kt(f"{tag}: GEMM keys and values", lambda: ops.linear_shallow(rows, ew), *gemm(R, H * 256, rank))
            written = ops.linear_shallow(rows, ew)
            for name, kw in (("latent attention, window + sinks, keys written out", dict(gate=None, **mine)),
                             ("[gisilix] latent attention, window + gate, keys written out", theirs)):
                kt(f"{tag}: {name}", lambda: ops.expanded_attention(fq, written, plan, cu, 0.07, window, n, out=yv, **kw),
                   T * H * (192 + d) * 2 + R * H * 320 * 2, 2.0 * pairs(window) * H * 320)
            del written, ew, rows, fq
        kt(f"{tag}: output gate", lambda: ops.output_gate(yv, proj[:, qr + rank + rot:], d), T * H * d * 6)
        gu = rn(T, 2 * ((8 * width // 3 + 127) // 128 * 128))
        kt(f"{tag}: silu x up", lambda: ops.act_and_mul(gu, "silu"), gu.numel() * 3)
        ids, table = i32([i % 1000 for i in range(T)]), rn(1000, width)
        kt(f"{tag}: embedding to fp32", lambda: ops.embed_residual(ids, table, 2.0), T * width * 6)
        assert K.check_status(dev) == 0
        del proj, pages, gu, wl, wu, qp
        torch.cuda.empty_cache()
    return kt.rows
