"""Prefill and decode throughput of a hybrid decoder beside its closest relative of the same width, depth, heads and
active parameters per token, and the kernels of both against their rooflines.

``python bench.py --model fuzuvik-bf16`` (beside a Llama shape), ``--model kipedra-bf16`` (beside a Fuzuvik shape; expert
kernels beside those of gated experts), ``--model gisilix-bf16`` (beside a DeepSeek shape, ``bench_latent``) and ``--model
sobivik-bf16`` (beside a Fuzuvik shape, ``bench_sobivik``) print one JSON line.  Weights are random; token rates are timed with CUDA
events around the model's forward (prefill) and around replays of its decode graph.  Kernels are timed one by one
with the L2 flushed in front of every launch; a roofline is the larger of bytes over the measured copy bandwidth and
FLOPs over the measured rate of the unit that does them (bf16 tensor cores, or fp32 FMA for the state recurrences).
"""
from __future__ import annotations

import json
import math
import os
from pathlib import Path

import numpy as np
import torch

FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12      # nominal: 128 fp32 FMA per SM and cycle


def peaks():
    f = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if f.exists():
        d = json.loads(f.read_text())
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def fuzuvik_like(width: int, layers: int, vocab: int, chunk: int) -> dict:
    from ..utils import synthetic as syn

    h, ff = width // 128, 4 * width
    kinds = [syn.fuzuvik_attention(h, h // 4, 128, 128, chunk, ff=ff, scaling=(8.0, 1.0, 4.0, 8192), base=500000.0),
             syn.fuzuvik_delta(h, h, 128, 128, 4, ff=ff),
             syn.fuzuvik_attention(h, h // 4, 128, 128, chunk, ff=ff, scaling=(8.0, 1.0, 4.0, 8192), base=500000.0),
             syn.fuzuvik_lightning(h, 128, 128, ff=ff)]
    return syn.fuzuvik_config([kinds[i % 4] for i in range(layers)], width=width, vocab=vocab, eps=1e-6)


def llama_like(width: int, layers: int, vocab: int) -> dict:
    from ..utils import synthetic as syn

    # a gated feed-forward of 8/3 width has the parameters of a plain one of 4 width
    return syn.llama_config(hidden=width, layers=layers, heads=width // 128, kv_heads=width // 512,
                            intermediate=(8 * width // 3 + 127) // 128 * 128, vocab=vocab, theta=500000.0, max_pos=16384)


def kipedra_like(width: int, layers: int, vocab: int, window: int) -> dict:
    """Every fourth layer dense, the others with 16 experts of which a token uses four: per token the parameters of a plain
    feed-forward of 4 x width."""
    from ..utils import synthetic as syn

    h = width // 128
    dense, moe = syn.kipedra_dense((8 * width // 3 + 127) // 128 * 128), syn.kipedra_moe(ff=width, experts=16, top=4, scale=1.0)
    attn = lambda mlp: syn.kipedra_attention(h, h // 4, 128, 128, window, base=500000.0, mlp=mlp)
    kinds = [attn(dense), syn.kipedra_delta(h, h, 128, 128, 4, mlp=moe), attn(moe), syn.kipedra_delta(h, h, 128, 128, 4, mlp=moe)]
    return syn.kipedra_config([kinds[i % 4] for i in range(layers)], width=width, vocab=vocab, eps=1e-6, residual_mult=0.3)


def fuzuvik_twin(width: int, layers: int, vocab: int, window: int) -> dict:
    """The Fuzuvik shape that ``kipedra_like`` is measured beside: attention and delta layers in turn, chunks as long as the
    windows, dense feed-forwards."""
    cfg = fuzuvik_like(width, layers, vocab, window)
    for i in range(3, layers, 4):
        cfg["layers"][i] = cfg["layers"][1]
    return cfg


def make_runner(cfg: dict, dev):
    from ..models.arch import ModelConfig
    from ..models.decoder import CausalDecoder
    from ..models.flash_causal_lm import FlashCausalLM
    from ..utils import synthetic as syn
    from ..utils.tokenizer import ByteTokenizer

    mc = ModelConfig(cfg)
    if cfg.get("architecture") or cfg["model_type"] == "deepseek_v2":
        from .bench_latent import deepseek_tensors

        kw = dict(dtype=torch.bfloat16, device=str(dev))
        tensors = {"Kipedra": lambda: syn.kipedra_state_dict(cfg, **kw), "Gisilix": lambda: syn.gisilix_state_dict(cfg, **kw),
                   "Sobivik": lambda: syn.sobivik_state_dict(cfg, **kw),
                   "Fuzuvik": lambda: syn.fuzuvik_state_dict(cfg, rank=128, **kw),
                   None: lambda: deepseek_tensors(cfg, dev)}[cfg.get("architecture")]()
        w = syn.DictWeights(tensors, dev, torch.bfloat16, bare_names=bool(cfg.get("architecture")))
        del tensors
    else:
        w = syn.SyntheticWeights(cfg, dev, torch.bfloat16)
    model = CausalDecoder(mc, w, max_positions=16384)
    return FlashCausalLM(model, ByteTokenizer(mc.vocab_size), torch.bfloat16, dev)


def timed(fn, steps: int, warmup: int) -> float:
    """Milliseconds per call."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


class Sequences:
    """Batch of sequences with pages and (for recurrent layers) slots, driven through the runner's metadata builder."""

    def __init__(self, runner, batch: int, ctx: int, vocab: int):
        from ..models.flash_causal_lm import BLOCK_SIZE, FlashCausalLMBatch, Seq
        from ..proto import generate_v3 as pb

        per = math.ceil((ctx + 16) / BLOCK_SIZE)
        runner.init_kv_cache(1 + batch * per, state_slots=batch)
        rng = np.random.default_rng(0)
        seqs = []
        for i in range(batch):
            blocks = list(range(1 + i * per, 1 + (i + 1) * per))
            slots = (np.asarray(blocks, dtype=np.int32)[:, None] * BLOCK_SIZE
                     + np.arange(BLOCK_SIZE, dtype=np.int32)[None]).reshape(-1)
            ids = rng.integers(3, vocab, size=ctx).tolist()
            seqs.append(Seq(request=pb.Request(id=i), ids=ids, prompt_len=ctx, cache_len=0, blocks=blocks, slots=slots,
                            stopping=None, top_n=0, prefix_offset=0, read_offset=0))
        self.runner, self.batch, self.ctx = runner, FlashCausalLMBatch(0, seqs, None, runner.device), ctx

    def prefill(self):
        meta, _ = self.runner.build_meta(self.batch, [self.ctx] * len(self.batch))
        return meta


def model_rates(cfg: dict, dev, vocab: int, prefills, decodes, steps: int, warmup: int) -> dict:
    from ..models.graphs import DecodeGraphs
    from . import cuda as K

    runner = make_runner(cfg, dev)
    out = {"prefill_tok_s": {}, "decode_tok_s": {}}
    for b, t in prefills:
        s = Sequences(runner, b, t, vocab)
        meta = s.prefill()
        ms = timed(lambda: runner.model.forward(meta, runner.kv_cache), max(3, steps // 4), warmup)
        out["prefill_tok_s"][f"{b}x{t}"] = round(b * t / ms * 1e3)
    for b, ctx in decodes:
        s = Sequences(runner, b, ctx, vocab)
        for q in s.batch.seqs:
            if runner.recurrent:
                runner.state_slot(q, 0)
            q.cache_len, q.prefilling = ctx - 1, False
        g = DecodeGraphs(runner, ctx + 16, buckets=[b])
        g.capture_all()
        g.run(s.batch, [1] * b)
        graph = g.buckets[b].graph
        ms = timed(graph.replay, steps, warmup)
        out["decode_tok_s"][f"{b}@{ctx}"] = round(b / ms * 1e3)
        del g, graph
    assert K.check_status(dev) == 0, "a kernel wait timed out"
    del runner
    torch.cuda.empty_cache()
    return out


class KernelTimer:
    def __init__(self, dev, iters: int = 12):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
        self.iters = iters
        self.hbm, self.tensor, self.source = peaks()
        self.rows = []

    def __call__(self, name: str, fn, bytes_: float, flops: float = 0.0, unit: str = "tensor"):
        for _ in range(3):
            fn()
        us = []
        for _ in range(self.iters):
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            us.append(a.elapsed_time(b) * 1e3)
        t = sorted(us)[len(us) // 2]
        rate = self.tensor if unit == "tensor" else FP32_TFLOPS * 1e12
        roof = max(bytes_ / self.hbm, flops / rate) * 1e6
        self.rows.append({"kernel": name, "us": round(t, 1), "roofline_us": round(roof, 1), "frac": round(roof / t, 3),
                          "bound": "bytes" if bytes_ / self.hbm >= flops / rate else unit})


def kernel_rows(dev, width: int, chunk: int, prefill, decode) -> list:
    """Every kernel of the design at layer size, and the like kernels of the Llama-shaped model."""
    from .. import ops
    from . import cuda as K
    from ..models.arch import MixerSpec
    from ..models.mixers import RotaryTables
    from ..utils.rotary import RotaryTable

    H, G, d = width // 128, width // 512, 128
    kt = KernelTimer(dev)
    bf = torch.bfloat16
    spec = MixerSpec("attention", H, G, d, d, rot_dims=d, rot_base=500000.0)
    tab = RotaryTables(16384, dev).get(spec).cos_sin
    taps = 4
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rn = lambda *s, dt=bf: torch.randn(*s, device=dev, dtype=torch.float32).to(dt)
    for label, B, n, ctx in [("prefill", *prefill, prefill[1]), ("decode", decode[0], 1, decode[1])]:
        T = B * n
        tag = f"{label} {B}x{n}" + (f" @{ctx}" if n == 1 else "")
        cu, kv, slots = i32([i * n for i in range(B + 1)]), i32([ctx] * B), i32(list(range(B)))
        per = math.ceil(ctx / 16)
        bt = torch.arange(B * per, dtype=torch.int32, device=dev).view(B, per)
        pos = i32([ctx - n + i for _ in range(B) for i in range(n)])
        page = i32([b * per * 16 + ctx - n + i for b in range(B) for i in range(n)])
        kc, vc = rn(B * per, 16, G, d), rn(B * per, 16, G, d)
        # ---- attention layer
        qw = (H + 2 * G) * d
        proj, first = rn(T, qw), rn(T, G * d)
        offs = [0, H * d, H * d + G * d]
        io = T * qw * 2 * 2
        kt(f"{tag}: rotate + unit rms + value mix + store", lambda: ops.rotate_norm_store(
            proj, offs, pos, tab, page, kc, vc, H, G, d, d, d, True, 1e-6, first, 0.3), io + T * G * d * 2)
        kt(f"{tag}: [llama] rope + store", lambda: ops.rope_and_cache(proj, pos, tab, page, kc, vc, H, G, d, d), io)
        q = rn(T, H, d)
        for c, nm in ((chunk, "attention, chunk + sink"), (0, "[llama] attention")):
            span = min(ctx, c) if c else ctx
            if n > 1:
                pairs = B * (sum(min(i % c + 1, i + 1) if c else i + 1 for i in range(n)))
                by, fl = T * H * d * 4 + 2 * T * G * d * 2, 4.0 * pairs * H * d
            else:
                span = (ctx - 1) % c + 1 if c else ctx
                by, fl = 2 * B * span * G * d * 2 + T * H * d * 4, 0.0
            kt(f"{tag}: {nm}", lambda: ops.paged_attention(q, kc, vc, bt, cu, kv, d ** -0.5, max_q=n, max_kv=ctx, chunk=c,
                                                           sink=bool(c)), by, fl)
        # ---- delta layer
        C = 3 * H * d
        cols = C + (H + 7) // 8 * 8 + 256
        x, a = rn(T, cols), rn(T, H * d)
        conv = ops.conv_weights([torch.randn(H * d, taps, device=dev) for _ in range(3)], dev)
        a_log, bias = torch.zeros(H, device=dev), torch.randn(H * d, device=dev) - 2
        cs, S = torch.zeros(B, taps - 1, C, dtype=bf, device=dev), torch.zeros(B, H, d, d, device=dev)
        do = [0, H * d, 2 * H * d, 3 * H * d]
        prep = lambda: ops.delta_inputs(x, do, a, conv, a_log, bias, cu, kv, slots, cs, H, H, d, d, d, n == 1)
        cbytes = B * (taps - 1) * C * 2 * (2 if n == 1 else 1)
        kt(f"{tag}: delta inputs (conv, norms, decays)", prep, T * H * d * (4 * 2 + 4 * 4) + cbytes)
        r = prep()
        st = B * H * d * d * 4 * (2 if n == 1 else 1)
        kt(f"{tag}: delta scan", lambda: ops.delta_scan(*r, cu, kv, slots, S, d, n), T * H * d * 4 * 5 + st,
           7.0 * T * H * d * d, "fp32")
        o = rn(T, H, d, dt=torch.float32)
        w1 = torch.ones(d, device=dev)
        kt(f"{tag}: norm x gate, per head", lambda: ops.gated_norm(o, a, w1, 1e-6, H, H * d), T * H * d * 8)
        # ---- fixed-decay layer
        dec = torch.full((H,), 0.99, device=dev)
        y = rn(T, 4 * H * d)
        kt(f"{tag}: decay scan", lambda: ops.decay_scan(y, [0, H * d, 2 * H * d], dec, cu, kv, slots, S, H, d, d, n),
           T * H * d * (3 * 2 + 4) + st, 5.0 * T * H * d * d, "fp32")
        w2 = torch.ones(H * d, device=dev)
        kt(f"{tag}: norm x gate, whole row", lambda: ops.gated_norm(o, y[:, 3 * H * d:], w2, 1e-6, 1, H * d), T * H * d * 8)
        # ---- common
        res, dl, w = rn(T, width, dt=torch.float32), rn(T, width), rn(width)
        kt(f"{tag}: residual (fp32) + norm", lambda: ops.residual_norm(dl, res, w, 1e-6), T * width * 12)
        rb = rn(T, width)
        kt(f"{tag}: [llama] residual (bf16) + norm", lambda: ops.rms_norm(dl, rb, w, 1e-6), T * width * 8)
        u = rn(T, 4 * width)
        kt(f"{tag}: gelu", lambda: ops.activation(u, "gelu"), T * 4 * width * 4)
        gu = rn(T, 2 * (8 * width // 3 // 128 * 128))
        kt(f"{tag}: [llama] silu x up", lambda: ops.act_and_mul(gu, "silu"), gu.numel() * 3)
        ids, table = i32([i % 1000 for i in range(T)]), rn(1000, width)
        kt(f"{tag}: embedding to fp32", lambda: ops.embed_residual(ids, table, 2.0), T * width * 6)
        wq = rn(cols, width)
        xw = rn(T, width)
        kt(f"{tag}: GEMM q k v b a1 g1", lambda: ops.linear(xw, wq), (T + cols) * width * 2 + T * cols * 2, 2.0 * T * cols * width)
        wl = rn(qw, width)
        kt(f"{tag}: [llama] GEMM q k v", lambda: ops.linear(xw, wl), (T + qw) * width * 2 + T * qw * 2, 2.0 * T * qw * width)
        w3 = rn(H * d, 128)
        kt(f"{tag}: GEMM a2 (rank 128)", lambda: ops.linear_shallow(x[:, C + (H + 7) // 8 * 8:][:, :128], w3),
           (T + H * d) * 256 + T * H * d * 2, 2.0 * T * H * d * 128)
        assert K.check_status(dev) == 0
        torch.cuda.empty_cache()
    return kt.rows


def kipedra_rows(dev, width: int, window: int, prefill, decode) -> list:
    """Every kernel of the design at layer size, and the like kernels of the Fuzuvik shape and of gated experts."""
    from .. import ops
    from . import cuda as K
    from ..models.arch import MixerSpec
    from ..models.mixers import RotaryTables

    H, G, d, taps = width // 128, width // 512, 128, 4
    kt = KernelTimer(dev)
    bf, f32 = torch.bfloat16, torch.float32
    tab = RotaryTables(16384, dev).get(MixerSpec("attention", H, G, d, d, rot_dims=d, rot_base=500000.0)).cos_sin
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rn = lambda *s, dt=bf: torch.randn(*s, device=dev, dtype=f32).to(dt)
    for label, B, n, ctx in [("prefill", *prefill, prefill[1]), ("decode", decode[0], 1, decode[1])]:
        T, one = B * n, n == 1
        tag = f"{label} {B}x{n}" + (f" @{ctx}" if one else "")
        cu, kv, slots = i32([i * n for i in range(B + 1)]), i32([ctx] * B), i32(list(range(B)))
        per = math.ceil(ctx / 16)
        bt = torch.arange(B * per, dtype=torch.int32, device=dev).view(B, per)
        pos = i32([ctx - n + i for _ in range(B) for i in range(n)])
        page = i32([b * per * 16 + ctx - n + i for b in range(B) for i in range(n)])
        kc, vc = rn(B * per, 16, G, d), rn(B * per, 16, G, d)
        # ---- attention layer
        qw = (H + 2 * G) * d
        proj, first, offs = rn(T, qw), rn(T, G * d), [0, H * d, H * d + G * d]
        past = torch.zeros(B, taps - 1, qw, dtype=bf, device=dev)
        conv = ops.ShortConv(ops.conv_weights([torch.randn(w * d, taps, device=dev) for w in (H, G, G)], dev), past, cu, kv, slots, one)
        io, pb = T * qw * 4, B * (taps - 1) * qw * 2 * (2 if one else 1)
        kt(f"{tag}: convolution + rotate + store", lambda: ops.rotate_norm_store(
            proj, offs, pos, tab, page, kc, vc, H, G, d, d, d, False, 1e-6, interleaved=True, conv=conv), io + pb)
        kt(f"{tag}: [fuzuvik] rotate + unit rms + value mix + store", lambda: ops.rotate_norm_store(
            proj, offs, pos, tab, page, kc, vc, H, G, d, d, d, True, 1e-6, first, 0.3), io + T * G * d * 2)
        q = rn(T, H, d)
        for name, kw in (("attention, window", dict(window=window)), ("[fuzuvik] attention, chunk + sink", dict(chunk=window, sink=True))):
            if one:
                span = min(ctx, window) if "window" in kw else (ctx - 1) % window + 1
                by, fl = 2 * B * span * G * d * 2 + T * H * d * 4, 0.0
            else:
                pairs = B * sum(min(i + 1, window) if "window" in kw else i % window + 1 for i in range(n))
                by, fl = T * H * d * 4 + 2 * T * G * d * 2, 4.0 * pairs * H * d
            kt(f"{tag}: {name}", lambda: ops.paged_attention(q, kc, vc, bt, cu, kv, d ** -0.5, max_q=n, max_kv=ctx, **kw), by, fl)
        wl, xw, bias = rn(qw, width), rn(T, width), rn(qw)
        kt(f"{tag}: GEMM q k v + bias", lambda: ops.linear(xw, wl, bias), (T + qw) * width * 2 + T * qw * 2, 2.0 * T * qw * width)
        kt(f"{tag}: [fuzuvik] GEMM q k v", lambda: ops.linear(xw, wl), (T + qw) * width * 2 + T * qw * 2, 2.0 * T * qw * width)
        # ---- delta layer
        C, hp = 3 * H * d, (H + 7) // 8 * 8
        cols = C + 2 * hp + H * d
        x, a = rn(T, cols), rn(T, H * d)
        taps_w = ops.conv_weights([torch.randn(H * d, taps, device=dev) for _ in range(3)], dev)
        a_log, bh, bc = torch.zeros(H, device=dev), torch.randn(H, device=dev) - 2, torch.randn(H * d, device=dev) - 2
        cs, S = torch.zeros(B, taps - 1, C, dtype=bf, device=dev), torch.zeros(B, H, d, d, device=dev)
        do = [0, H * d, 2 * H * d, C, C + hp, C + 2 * hp]
        cb, st = B * (taps - 1) * C * 2 * (2 if one else 1), B * H * d * d * 4 * (2 if one else 1)
        prep = lambda: ops.delta_inputs(x, do, x[:, do[4]:do[4] + H], taps_w, a_log, bh, cu, kv, slots, cs, H, H, d, d, d, one, True)
        wide = lambda: ops.delta_inputs(x, do, a, taps_w, a_log, bc, cu, kv, slots, cs, H, H, d, d, d, one)
        kt(f"{tag}: delta inputs, decay per head", prep, T * H * (d * (3 * 2 + 3 * 4) + 16) + cb)
        kt(f"{tag}: [fuzuvik] delta inputs", wide, T * H * d * (4 * 2 + 4 * 4) + cb)
        r = prep()
        kt(f"{tag}: delta scan, decay per head", lambda: ops.delta_scan(*r, cu, kv, slots, S, d, n), T * H * (d * 16 + 8) + st,
           7.0 * T * H * d * d, "fp32")
        r2 = wide()
        kt(f"{tag}: [fuzuvik] delta scan", lambda: ops.delta_scan(*r2, cu, kv, slots, S, d, n), T * H * d * 20 + st,
           7.0 * T * H * d * d, "fp32")
        del r2
        o, w1 = rn(T, H, d, dt=f32), torch.ones(d, device=dev)
        kt(f"{tag}: norm x silu gate", lambda: ops.gated_norm(o, x[:, do[5]:], w1, 1e-6, H, H * d, "silu"), T * H * d * 8)
        kt(f"{tag}: [fuzuvik] norm x gate", lambda: ops.gated_norm(o, a, w1, 1e-6, H, H * d), T * H * d * 8)
        wq = rn(cols, width)
        kt(f"{tag}: GEMM q k v b a g", lambda: ops.linear(xw, wq), (T + cols) * width * 2 + T * cols * 2, 2.0 * T * cols * width)
        # ---- stream
        res, d1, d2, n1, n2 = rn(T, width, dt=f32), rn(T, width), rn(T, width), rn(width), rn(width)
        kt(f"{tag}: residual (fp32, two outputs) + two norms", lambda: ops.residual_norm(
            (d1, d2), res, n1, 1e-6, scale=0.3, unit_offset=True, weight2=n2), T * width * 16)
        kt(f"{tag}: [fuzuvik] residual (fp32) + norm", lambda: ops.residual_norm(d1, res, n1, 1e-6), T * width * 12)
        # ---- feed-forwards
        ff = (8 * width // 3 + 127) // 128 * 128
        gu, u = rn(T, 2 * ff), rn(T, 4 * width)
        kt(f"{tag}: gelu x up", lambda: ops.act_and_mul(gu, "gelu_tanh"), gu.numel() * 3)
        kt(f"{tag}: [llama] silu x up", lambda: ops.act_and_mul(gu, "silu"), gu.numel() * 3)
        kt(f"{tag}: [fuzuvik] gelu", lambda: ops.activation(u, "gelu"), u.numel() * 4)
        del gu, u
        E, top, I = 16, 4, width
        rw, corr = rn(E, width) * 0.02, torch.zeros(E, device=dev)
        rb = (T + E) * width * 2 + T * top * 8
        route = lambda: ops.moe_route_sigmoid(xw, rw, corr, top, 1.0)
        kt(f"{tag}: router (sigmoid, fp32)", route, rb, 2.0 * T * E * width)
        kt(f"{tag}: [mixtral] router (softmax)", lambda: ops.moe_topk_softmax(ops.linear(xw, rw), top), rb, 2.0 * T * E * width)
        tw, ti = route()
        up, down, used = rn(E, I, width) * 0.02, rn(E, width, I) * 0.02, min(E, T * top)
        kt(f"{tag}: experts, ungated", lambda: ops.moe_plain_experts(xw, up, down, tw, ti, "relu2"),
           used * 2 * I * width * 2 + T * width * 4, 4.0 * T * top * I * width)
        wgu, wd = rn(E, I, width) * 0.02, rn(E, width, I // 2) * 0.02
        kt(f"{tag}: [mixtral] experts, gated, half as wide", lambda: ops.moe_experts(xw, wgu, wd, tw, ti, "silu"),
           used * 3 * (I // 2) * width * 2 + T * width * 4, 3.0 * T * top * I * width)
        assert K.check_status(dev) == 0
        del up, down, wgu, wd
        torch.cuda.empty_cache()
    return kt.rows


def run(args, clock_sampler) -> int:
    from . import cuda as K
    from .bench_latent import deepseek_like, gisilix_like, gisilix_rows
    from .bench_sobivik import fuzuvik_relative, sobivik_like, sobivik_rows

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    K.load()
    vocab, layers = 32000, args.layers or 8
    # model, its relative, kernels, window or chunk, (batch, context) of the decode steps both run and of those it runs alone
    name, own, other, twin, rows_of, span, decodes, alone = {
        "fuzuvik-bf16": ("fuzuvik", fuzuvik_like, "llama", lambda w, n, v, s: llama_like(w, n, v), kernel_rows, 8192, [(16, 2048), (256, 2048)], []),
        "kipedra-bf16": ("kipedra", kipedra_like, "fuzuvik", fuzuvik_twin, kipedra_rows, 1024, [(16, 2048), (256, 2048)], []),
        # 256 x 2048 tokens of keys and values per head do not fit beside the weights
        "gisilix-bf16": ("gisilix", gisilix_like, "deepseek", lambda w, n, v, s: deepseek_like(w, n, v), gisilix_rows, 1024,
                         [(16, 2048), (64, 2048)], [(256, 2048)]),
        "sobivik-bf16": ("sobivik", sobivik_like, "fuzuvik", fuzuvik_relative, sobivik_rows, 1024, [(16, 2048), (256, 2048)], []),
    }[args.model]
    sampler = clock_sampler(0)
    sampler.start()
    sizes = {}
    prefills = [(4, 2048), (1, 8192)]
    for width in (2048, 4096):
        cfgs = {name: own(width, layers, vocab, span), other: twin(width, layers, vocab, span)}
        sizes[str(width)] = {k: model_rates(c, dev, vocab, prefills, decodes + (alone if k == name else []), args.steps, args.warmup)
                             for k, c in cfgs.items()}
    batch = (decodes + alone)[-1][0]
    rows = rows_of(dev, 4096, span, (4, 2048), (decodes[-1][0], 2048))
    clocks = sampler.stop()
    value = sizes["4096"][name]["decode_tok_s"][f"{batch}@2048"]
    print(json.dumps({
        "metric": f"output tok/s (decode, {args.model})", "value": value, "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
        "warmup": args.warmup, "ms_per_step": round(batch * 1e3 / value, 4), "higher_is_better": True, "scaling": "strong",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random tokens, random weights", "impl": "b200",
        "config": {"model": f"{name}-{layers}L", "global_batch": batch, "seq_len": 2048, "chunk" if name == "fuzuvik" else "window": span,
                   "parallelism": "tp1", "l2": "models: inputs larger than L2; kernels: L2 flushed before every launch"},
        "sizes": sizes, "kernels": rows, "peaks": peaks()[2], "clocks": clocks}), flush=True)
    return 0
