"""Shapes and kernels of ``python bench.py --model gisilix-bf16`` (see ``bench_hybrid``): a Gisilix decoder beside a
DeepSeek-V2 shape with the same latent attention sizes, width, depth and active parameters per token."""
from __future__ import annotations

import math
from typing import Dict

import torch


def gisilix_like(width: int, layers: int, vocab: int, window: int) -> dict:
    """Heads of 128 (+ 64 rotated), latents of 512; every second layer routed: 16 experts of which a token uses four, beside
    a shared one."""
    from ..utils import synthetic as syn

    h, ff = width // 128, width // 2
    dense, moe = syn.kipedra_dense(5 * ff), syn.gisilix_moe(ff, 16, 4, ff)
    attn = lambda src, mlp: syn.gisilix_attention(h, h // 4, 128, 128, 0.1, 4096, 30.0, kv_from=src, mlp=mlp)
    kinds = lambda i: [attn(None, dense),
                       syn.gisilix_rotated_latent(h, 128, 128, 512, 64, window, 500000.0, (8.0, 32.0, 1.0, 4096), mlp=moe),
                       syn.gisilix_latent(h, 128, 128, 512, mlp=dense), attn(i - i % 4, moe)][i % 4]
    return syn.gisilix_config([kinds(i) for i in range(layers)], width=width, vocab=vocab, eps=1e-6)


def deepseek_like(width: int, layers: int, vocab: int) -> dict:
    h, ff = width // 128, width // 2
    return dict(model_type="deepseek_v2", hidden_size=width, num_hidden_layers=layers, num_attention_heads=h, vocab_size=vocab,
                qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, kv_lora_rank=512, q_lora_rank=None, intermediate_size=5 * ff,
                moe_intermediate_size=ff, n_routed_experts=16, n_shared_experts=1, num_experts_per_tok=4, first_k_dense_replace=0,
                moe_layer_freq=2, norm_topk_prob=True, hidden_act="silu", rms_norm_eps=1e-6, rope_theta=500000.0,
                max_position_embeddings=16384)


def deepseek_tensors(cfg: dict, device) -> Dict[str, torch.Tensor]:
    W, H, V, ff = cfg["hidden_size"], cfg["num_attention_heads"], cfg["vocab_size"], cfg["moe_intermediate_size"]
    rnd = lambda *s: (torch.randn(*s, device=device) * s[-1] ** -0.5).to(torch.bfloat16)
    ones = lambda n: torch.ones(n, dtype=torch.bfloat16, device=device)
    sd = {"model.embed_tokens.weight": rnd(V, W), "lm_head.weight": rnd(V, W), "model.norm.weight": ones(W)}

    def feed_forward(p, width):
        sd.update({f"{p}.gate_proj.weight": rnd(width, W), f"{p}.up_proj.weight": rnd(width, W), f"{p}.down_proj.weight": rnd(W, width)})

    for i in range(cfg["num_hidden_layers"]):
        p = f"model.layers.{i}"
        a = f"{p}.self_attn"
        sd.update({f"{p}.input_layernorm.weight": ones(W), f"{p}.post_attention_layernorm.weight": ones(W), f"{a}.q_proj.weight": rnd(H * 192, W),
                   f"{a}.kv_a_proj_with_mqa.weight": rnd(576, W), f"{a}.kv_a_layernorm.weight": ones(512), f"{a}.kv_b_proj.weight": rnd(H * 256, 512),
                   f"{a}.o_proj.weight": rnd(W, H * 128)})
        if i % 2:
            feed_forward(f"{p}.mlp", cfg["intermediate_size"])
            continue
        sd[f"{p}.mlp.gate.weight"] = rnd(16, W)
        for e in range(16):
            feed_forward(f"{p}.mlp.experts.{e}", ff)
        feed_forward(f"{p}.mlp.shared_experts", ff)
    return sd


def gisilix_rows(dev, width: int, window: int, prefill, decode) -> list:
    """Every kernel of the design at layer size, and the like kernels of the DeepSeek and Llama shapes."""
    import numpy as np

    from .. import ops
    from . import cuda as K
    from ..models.arch import MixerSpec
    from ..models.mixers import Expansion, RotaryTables, plan_expansion
    from .bench_hybrid import KernelTimer

    H, G, d, rank, rot = width // 128, width // 512, 128, 512, 64
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
        cu, kv = i32([i * n for i in range(B + 1)]), i32([ctx] * B)
        per = math.ceil(ctx / 16)
        bt = torch.arange(B * per, dtype=torch.int32, device=dev).view(B, per)
        pos = i32([ctx - n + i for _ in range(B) for i in range(n)])
        page = i32([b * per * 16 + ctx - n + i for b in range(B) for i in range(n)])
        pairs = lambda w: B * sum(min(i + 1, w) if w else i + 1 for i in range(ctx - n, ctx))
        seen = lambda w: B * min(ctx, w + n - 1 if w else ctx)
        xw = rn(T, width)
        # ---- attention with row norms
        qw = (2 * H + 2 * G) * d
        proj, offs = rn(T, qw), [0, H * d, (H + G) * d, (H + 2 * G) * d]
        kc, vc = rn(B * per, 16, G, d), rn(B * per, 16, G, d)
        wq, wk, sink = torch.ones(H * d, device=dev), torch.ones(G * d, device=dev), torch.zeros(H, device=dev)
        io = T * (H + 2 * G) * d * 4
        kt(f"{tag}: row norms + temperature + store", lambda: ops.row_norm_store(
            proj, offs, pos, page, kc, vc, wq, wk, 1e-6, H, G, d, d, d, (0.1, 4096)), io)
        kt(f"{tag}: [llama] rope + store", lambda: ops.rope_and_cache(proj[:, :(H + 2 * G) * d].contiguous() if one else proj[:, :(H + 2 * G) * d],
                                                                      pos, full_tab, page, kc, vc, H, G, d, d), io)
        q = rn(T, H, d)
        by, fl = (seen(0) * 2 * G + 2 * T * H) * d * 2, 4.0 * pairs(0) * H * d
        kt(f"{tag}: attention, cap + sink", lambda: ops.paged_attention(q, kc, vc, bt, cu, kv, d ** -0.5, softcap=30.0, max_q=n, max_kv=ctx,
                                                                        sink=sink), by, fl)
        kt(f"{tag}: [llama] attention", lambda: ops.paged_attention(q, kc, vc, bt, cu, kv, d ** -0.5, max_q=n, max_kv=ctx), by, fl)
        kt(f"{tag}: output gate", lambda: ops.output_gate(q, proj[:, offs[3]:], d), T * H * d * 6)
        w = rn(qw, width)
        kt(f"{tag}: GEMM q k v g", lambda: ops.linear(xw, w), *gemm(T, qw, width))
        del kc, vc, w
        # ---- latent attention
        cols = H * (d + rot) + rank + rot + H
        off, wide = ops.latent_layout(rank, rot, bf, dev)
        proj, pages, norm = rn(T, cols), rn(B * per, 16, 1, wide), torch.ones(rank, device=dev)
        w = rn(cols, width)
        kt(f"{tag}: GEMM q dkv g", lambda: ops.linear(xw, w), *gemm(T, cols, width))
        gate = proj[:, cols - H:]
        for win, name in ((0, "latent attention"), (window, "latent attention, window + gate")):
            g = gate if win else None
            if one:
                lq = rn(T, H, wide)
                a = ops.latent_attention(lq, pages, rank, bt, cu, kv, 0.07, win or -1, 1, ctx, g)
                kt(f"{tag}: {name}", lambda: ops.latent_attention(lq, pages, rank, bt, cu, kv, 0.07, win or -1, 1, ctx, g),
                   seen(win) * wide * 2 + T * H * (wide + rank) * 2, 2.0 * pairs(win) * H * (wide + rank))
                continue
            fq, o = rn(T, H, 192), torch.empty(T, H, d, dtype=bf, device=dev)
            arrays, scalars = plan_expansion(win, [0] * B, [n] * B, [np.arange(b * per * 16, (b + 1) * per * 16, dtype=np.int32) for b in range(B)])
            plan = Expansion(*(torch.from_numpy(x).to(dev) for x in arrays), *scalars)
            R = plan.rows.numel()
            if not win:
                ew = rn(H * 320, wide, std=0.05)
                rows = pages.view(-1, wide).index_select(0, plan.rows)
                kt(f"{tag}: gather of latent rows", lambda: pages.view(-1, wide).index_select(0, plan.rows), R * wide * 4)
                kt(f"{tag}: GEMM keys and values", lambda: ops.linear_shallow(rows, ew), *gemm(R, H * 256, rank))
                written = ops.linear_shallow(rows, ew)
            kt(f"{tag}: {name}, keys written out", lambda: ops.expanded_attention(fq, written, plan, cu, 0.07, win or -1, n, g, o),
               T * H * (192 + d) * 2 + R * H * 320 * 2, 2.0 * pairs(win) * H * 320)
            if win:
                lq = rn(T, H, wide)
                kt(f"{tag}: {name}, on latents", lambda: ops.latent_attention(lq, pages, rank, bt, cu, kv, 0.07, win, n, ctx, g),
                   T * H * (wide + rank) * 2 + R * wide * 2, 2.0 * pairs(win) * H * 320)
        if one:
            uk, uv = rn(H, d, rank), rn(H, d, rank)
            plain = proj[:, :H * (d + rot)].view(T, H, -1)[..., :d]
            kt(f"{tag}: latent norm + rotations + store", lambda: ops.latent_store(
                proj, H * (d + rot), norm, 1e-6, pos, tab, page, pages, lq, off, rank, rot, H, d), T * (H * rot + rank + rot) * 4)
            kt(f"{tag}: queries x key up-projection", lambda: torch.bmm(plain.transpose(0, 1), uk, out=lq[..., :off].transpose(0, 1)),
               H * d * rank * 2 + T * H * (d + rank) * 2, 2.0 * T * H * d * rank)
            y = torch.empty(T, H, d, dtype=bf, device=dev)
            kt(f"{tag}: outputs x value up-projection", lambda: torch.bmm(a.transpose(0, 1), uv.transpose(1, 2), out=y.transpose(0, 1)),
               H * d * rank * 2 + T * H * (d + rank) * 2, 2.0 * T * H * d * rank)
        else:
            kt(f"{tag}: latent norm + rotations + store", lambda: ops.latent_store(
                proj, H * (d + rot), norm, 1e-6, pos, tab, page, pages, None, off, rank, rot, H, d, fq), T * (2 * H * (d + rot) + 2 * (rank + rot)) * 2)
            del written, ew, rows
        # the like steps of the DeepSeek shape: latent expanded per head, heads of 256, every head's keys and values in pages
        kc, vc = (torch.zeros(B * per, 16, H, 256, dtype=bf, device=dev) for _ in range(2))
        c, kvb, pe, dq = rn(T, rank), rn(H * 256, rank), rn(T, rot), rn(T, H, 192)

        def assemble():
            both = ops.linear(c, kvb).view(T, H, 256)
            fused = c.new_zeros(T, 3 * H, 256)
            fused[:, :H, :rot], fused[:, :H, rot:192] = dq[..., d:], dq[..., :d]
            fused[:, H:2 * H, :rot], fused[:, H:2 * H, rot:192] = pe.unsqueeze(1), both[..., :d]
            fused[:, 2 * H:, :d] = both[..., d:]
            return ops.rope_and_cache(fused.view(T, -1), pos, tab, page, kc, vc, H, H, 256, rot, False)

        kt(f"{tag}: [deepseek] keys, values, rotations, store", assemble,
           H * 256 * rank * 2 + T * (H * 192 * 2 + rank + rot + H * 320) * 2, 2.0 * T * H * 256 * rank)
        q = assemble()
        kt(f"{tag}: [deepseek] attention", lambda: ops.paged_attention(q, kc, vc, bt, cu, kv, 0.07, max_q=n, max_kv=ctx),
           (seen(0) * H * 320 + T * H * 320) * 2, 2.0 * pairs(0) * H * 320)
        del kc, vc, q
        # ---- stream and feed-forward
        res, dl, nw = rn(T, width, dt=f32), rn(T, width), rn(width)
        kt(f"{tag}: residual (fp32, two outputs) + layer norm", lambda: ops.residual_norm((dl, xw), res, nw, 1e-6, layer=True, bias=nw), T * width * 14)
        rb = rn(T, width)
        kt(f"{tag}: [deepseek] residual (bf16) + norm", lambda: ops.rms_norm(dl, rb, nw, 1e-6), T * width * 8)
        gu = rn(T, 5 * width)
        kt(f"{tag}: silu x up", lambda: ops.act_and_mul(gu, "silu"), gu.numel() * 3)
        E, top, I = 16, 4, width // 2
        rw, bias, rbytes = rn(E, width, std=0.02), torch.zeros(E, device=dev), (T + E) * width * 2 + T * top * 8
        route = lambda: ops.moe_route_softmax(xw, rw, bias, top)
        kt(f"{tag}: router (fp32, softmax over the chosen)", route, rbytes, 2.0 * T * E * width)
        kt(f"{tag}: [mixtral] router", lambda: ops.moe_topk_softmax(ops.linear(xw, rw), top), rbytes, 2.0 * T * E * width)
        tw, ti = route()
        wu, wd = rn(E, 2 * I, width, std=0.02), rn(E, width, I, std=0.02)
        eb, ef = min(E, T * top) * 3 * I * width * 2 + T * width * 4, 6.0 * T * top * I * width
        kt(f"{tag}: experts", lambda: ops.moe_plain_experts(xw, wu, wd, tw, ti, "silu", True), eb, ef)
        kt(f"{tag}: [deepseek] experts", lambda: ops.moe_experts(xw, wu, wd, tw, ti, "silu"), eb, ef)
        assert K.check_status(dev) == 0
        del wu, wd, pages, proj
        torch.cuda.empty_cache()
    return kt.rows
