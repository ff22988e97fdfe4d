"""Random-weight checkpoints of a given architecture (tests, smoke run, benchmarks).

``write_llama_checkpoint`` writes an HF-layout directory (``config.json`` + ``model.safetensors``)
with weights ``N(0, std)`` from a seed and norm weights 1.0 — small models for CPU tests.
``SyntheticWeights`` generates an *in-memory* checkpoint tensor by tensor directly on the GPU for
benchmark-size models that would take too long to write to disk; it returns a ``Weights``-like
object the decoder loads from (same names, same sharding entry points).
"""
from __future__ import annotations

import json
import os
from pathlib import Path
from typing import Dict, Optional

import torch

from .weights import save_safetensors


def llama_config(hidden=256, layers=2, heads=4, kv_heads=2, intermediate=688, vocab=32000, eps=1e-5,
                 theta=10000.0, max_pos=4096, tie=False, model_type="llama", **extra) -> dict:
    cfg = dict(
        architectures=["LlamaForCausalLM"], model_type=model_type, hidden_size=hidden, num_hidden_layers=layers,
        num_attention_heads=heads, num_key_value_heads=kv_heads, intermediate_size=intermediate,
        vocab_size=vocab, rms_norm_eps=eps, rope_theta=theta, max_position_embeddings=max_pos,
        hidden_act="silu", tie_word_embeddings=tie, torch_dtype="float32", bos_token_id=1, eos_token_id=2,
    )
    cfg.update(extra)
    return cfg


def llama_state_dict(cfg: dict, seed: int = 0, std: float = 0.02, dtype=torch.float32,
                     device: str = "cpu") -> Dict[str, torch.Tensor]:
    """Random weights of a Llama / Mixtral shape as a CPU state dict; ``device`` is where the random numbers are
    drawn (a GPU draws a multi-billion-parameter checkpoint in seconds)."""
    g = torch.Generator(device=device).manual_seed(seed)
    H, L = cfg["hidden_size"], cfg["num_hidden_layers"]
    nh, nkv = cfg["num_attention_heads"], cfg["num_key_value_heads"]
    D = cfg.get("head_dim") or H // nh
    I, V = cfg["intermediate_size"], cfg["vocab_size"]

    def rnd(*shape):
        return (torch.randn(*shape, generator=g, device=device) * std).to(dtype).cpu()

    sd = {"model.embed_tokens.weight": rnd(V, H), "model.norm.weight": torch.ones(H, dtype=dtype)}
    if not cfg.get("tie_word_embeddings"):
        sd["lm_head.weight"] = rnd(V, H)
    E = cfg.get("num_local_experts", 0)
    for i in range(L):
        p = f"model.layers.{i}"
        sd[f"{p}.input_layernorm.weight"] = torch.ones(H, dtype=dtype)
        sd[f"{p}.post_attention_layernorm.weight"] = torch.ones(H, dtype=dtype)
        sd[f"{p}.self_attn.q_proj.weight"] = rnd(nh * D, H)
        sd[f"{p}.self_attn.k_proj.weight"] = rnd(nkv * D, H)
        sd[f"{p}.self_attn.v_proj.weight"] = rnd(nkv * D, H)
        sd[f"{p}.self_attn.o_proj.weight"] = rnd(H, nh * D)
        if cfg.get("attention_bias") or cfg["model_type"] == "qwen2":
            sd[f"{p}.self_attn.q_proj.bias"] = rnd(nh * D)
            sd[f"{p}.self_attn.k_proj.bias"] = rnd(nkv * D)
            sd[f"{p}.self_attn.v_proj.bias"] = rnd(nkv * D)
        if E:
            sd[f"{p}.block_sparse_moe.gate.weight"] = rnd(E, H)
            for e in range(E):
                sd[f"{p}.block_sparse_moe.experts.{e}.w1.weight"] = rnd(I, H)
                sd[f"{p}.block_sparse_moe.experts.{e}.w3.weight"] = rnd(I, H)
                sd[f"{p}.block_sparse_moe.experts.{e}.w2.weight"] = rnd(H, I)
        else:
            sd[f"{p}.mlp.gate_proj.weight"] = rnd(I, H)
            sd[f"{p}.mlp.up_proj.weight"] = rnd(I, H)
            sd[f"{p}.mlp.down_proj.weight"] = rnd(H, I)
    return sd


def write_llama_checkpoint(path, cfg: Optional[dict] = None, seed: int = 0, std: float = 0.02,
                           dtype=torch.float32, device: str = "cpu") -> Path:
    cfg = cfg or llama_config()
    p = Path(path)
    p.mkdir(parents=True, exist_ok=True)
    (p / "config.json").write_text(json.dumps(cfg, indent=1))
    save_safetensors(llama_state_dict(cfg, seed, std, dtype, device), p / "model.safetensors", {"format": "pt"})
    return p


def reference_llama_forward(sd: Dict[str, torch.Tensor], cfg: dict, input_ids: torch.Tensor) -> torch.Tensor:
    """Plain dense PyTorch Llama forward (no paging, no fusion) over one sequence ``input_ids[T]``.

    Independent oracle for the engine's logits: returns ``[T, vocab]`` in fp32.
    """
    H, L = cfg["hidden_size"], cfg["num_hidden_layers"]
    nh, nkv = cfg["num_attention_heads"], cfg["num_key_value_heads"]
    D = cfg.get("head_dim") or H // nh
    eps, theta = cfg["rms_norm_eps"], cfg["rope_theta"]
    T = input_ids.shape[0]
    x = sd["model.embed_tokens.weight"].float()[input_ids]
    pos = torch.arange(T, dtype=torch.float32)
    inv = 1.0 / (theta ** (torch.arange(0, D, 2, dtype=torch.float32) / D))
    ang = torch.outer(pos, inv)
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]

    def norm(v, w):
        return v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps) * w.float()

    def rope(v):
        a, b = v[..., : D // 2], v[..., D // 2:]
        return torch.cat([a * cos - b * sin, b * cos + a * sin], -1)

    mask = torch.full((T, T), float("-inf")).triu(1)
    for i in range(L):
        p = f"model.layers.{i}"
        h = norm(x, sd[f"{p}.input_layernorm.weight"])
        q = (h @ sd[f"{p}.self_attn.q_proj.weight"].float().t()).view(T, nh, D)
        k = (h @ sd[f"{p}.self_attn.k_proj.weight"].float().t()).view(T, nkv, D)
        v = (h @ sd[f"{p}.self_attn.v_proj.weight"].float().t()).view(T, nkv, D)
        q, k = rope(q), rope(k)
        k = k.repeat_interleave(nh // nkv, 1)
        v = v.repeat_interleave(nh // nkv, 1)
        att = torch.einsum("thd,shd->hts", q, k) / (D ** 0.5) + mask
        o = torch.einsum("hts,shd->thd", att.softmax(-1), v).reshape(T, nh * D)
        x = x + o @ sd[f"{p}.self_attn.o_proj.weight"].float().t()
        h = norm(x, sd[f"{p}.post_attention_layernorm.weight"])
        g = h @ sd[f"{p}.mlp.gate_proj.weight"].float().t()
        u = h @ sd[f"{p}.mlp.up_proj.weight"].float().t()
        x = x + (torch.nn.functional.silu(g) * u) @ sd[f"{p}.mlp.down_proj.weight"].float().t()
    x = norm(x, sd["model.norm.weight"])
    head = sd.get("lm_head.weight", sd["model.embed_tokens.weight"]).float()
    return x @ head.t()


# ---------------------------------------------------------------------------------------------
# benchmark-size models: weights generated on the device, shard by shard, never materialised whole
# ---------------------------------------------------------------------------------------------
class _GeneratedSlice:
    """Stands in for ``weights.TensorSlice``: produces (a slice of) a random tensor on demand.

    The values of rows ``[a, b)`` depend only on ``(name, dim, a)``, so a weight shard and the
    block scales computed from the same rows agree with each other.
    """

    def __init__(self, owner: "SyntheticWeights", name: str, shape, kind: str):
        self.owner, self.name, self.shape, self.kind = owner, name, tuple(shape), kind

    def get_shape(self):
        return self.shape

    def tensor(self):
        return self.slice_dim(0, 0, self.shape[0]) if self.shape else self.owner._make(self.name, self.kind, (), 0, 0)

    def slice_dim(self, dim: int, start: int, stop: int):
        shape = list(self.shape)
        shape[dim] = max(0, stop - start)
        return self.owner._make(self.name, self.kind, tuple(shape), dim, start)


class SyntheticWeights:
    """``Weights``-compatible provider of random Llama-architecture parameters created on the device.

    ``fp8_block=True`` serves every linear projection as e4m3 with ``weight_scale_inv`` per 128x128
    block, quantised from seeded ``N(0, std)`` bf16 values; embeddings, norms and the head stay bf16.
    """

    def __new__(cls, cfg: dict, device, dtype=torch.bfloat16, process_group=None, fp8_block: bool = False,
                std: float = 0.02, seed: int = 0):
        from .weights import Weights

        class _Impl(Weights):
            pass

        self = _Impl.__new__(_Impl)
        Weights.__init__(self, [], device, dtype, process_group=process_group)
        self.cfg, self.fp8_block, self.std, self.seed = cfg, fp8_block, std, seed
        H, L = cfg["hidden_size"], cfg["num_hidden_layers"]
        nh, nkv = cfg["num_attention_heads"], cfg["num_key_value_heads"]
        D = cfg.get("head_dim") or H // nh
        I, V = cfg["intermediate_size"], cfg["vocab_size"]
        E = cfg.get("num_local_experts", 0)
        shapes = {"model.embed_tokens.weight": ((V, H), "plain"), "model.norm.weight": ((H,), "ones"),
                  "lm_head.weight": ((V, H), "plain")}
        for i in range(L):
            p = f"model.layers.{i}"
            shapes[f"{p}.input_layernorm.weight"] = ((H,), "ones")
            shapes[f"{p}.post_attention_layernorm.weight"] = ((H,), "ones")
            lin = {f"{p}.self_attn.q_proj": (nh * D, H), f"{p}.self_attn.k_proj": (nkv * D, H),
                   f"{p}.self_attn.v_proj": (nkv * D, H), f"{p}.self_attn.o_proj": (H, nh * D)}
            if E:
                shapes[f"{p}.block_sparse_moe.gate.weight"] = ((E, H), "plain")
                for e in range(E):
                    lin[f"{p}.block_sparse_moe.experts.{e}.w1"] = (I, H)
                    lin[f"{p}.block_sparse_moe.experts.{e}.w3"] = (I, H)
                    lin[f"{p}.block_sparse_moe.experts.{e}.w2"] = (H, I)
            else:
                lin.update({f"{p}.mlp.gate_proj": (I, H), f"{p}.mlp.up_proj": (I, H), f"{p}.mlp.down_proj": (H, I)})
            for name, shp in lin.items():
                if fp8_block and not E:
                    shapes[f"{name}.weight"] = (shp, "fp8")
                    shapes[f"{name}.weight_scale_inv"] = (((shp[0] + 127) // 128, (shp[1] + 127) // 128), "scale")
                else:
                    shapes[f"{name}.weight"] = (shp, "plain")
        self._shapes = shapes
        self.routing = {k: 0 for k in shapes}

        def _slice(name, _self=self):
            h, real = _self.resolve(name)
            shp, kind = _self._shapes[real]
            return _GeneratedSlice(_self, real, shp, kind)

        def resolve(name, _self=self):
            if name in _self._shapes:
                return None, name
            raise KeyError(f"weight {name} does not exist")

        def _make(name, kind, shape, dim, start, _self=self):
            import zlib

            dev = _self.device
            if kind == "ones":
                return torch.ones(shape, dtype=_self.dtype, device=dev)
            base = name[: -len("_scale_inv")] if kind == "scale" else name
            row0 = start * (128 if kind == "scale" else 1)
            g = torch.Generator(device=dev)
            g.manual_seed((zlib.crc32(base.encode()) * 1000003 + dim * 7919 + row0 + _self.seed) & 0x7FFFFFFF)
            if kind == "plain":
                return (torch.randn(shape, generator=g, device=dev, dtype=torch.float32) * _self.std).to(_self.dtype)
            from ..ops import reference as ref

            if kind == "fp8":
                w = (torch.randn(shape, generator=g, device=dev, dtype=torch.float32) * _self.std).to(torch.bfloat16)
                if dim == 1 and shape[0] > 0:
                    pass
                q, _ = ref.fp8_quant_block_weight(w)
                return q
            # scale: regenerate the rows the scales belong to
            full_w = _self._shapes[base][0]
            wshape = list(full_w)
            wshape[dim] = shape[dim] * 128
            wshape[dim] = min(wshape[dim], full_w[dim] - row0)
            w = (torch.randn(tuple(wshape), generator=g, device=dev, dtype=torch.float32) * _self.std).to(torch.bfloat16)
            _, s = ref.fp8_quant_block_weight(w)
            return s

        self._slice = _slice
        self.resolve = resolve
        self._make = _make
        self.has_tensor = lambda name, _self=self: name in _self._shapes
        return self


def llama3_8b_config(**kw) -> dict:
    return llama_config(hidden=4096, layers=32, heads=32, kv_heads=8, intermediate=14336, vocab=128256,
                        theta=500000.0, max_pos=8192, **kw)


def llama3_70b_config(block_fp8: bool = True, **kw) -> dict:
    cfg = llama_config(hidden=8192, layers=80, heads=64, kv_heads=8, intermediate=28672, vocab=128256,
                       theta=500000.0, max_pos=8192, **kw)
    if block_fp8:
        cfg["quantization_config"] = {"quant_method": "fp8", "weight_block_size": [128, 128],
                                      "activation_scheme": "dynamic", "fmt": "e4m3"}
    return cfg


def mixtral_8x7b_config(**kw) -> dict:
    return llama_config(hidden=4096, layers=32, heads=32, kv_heads=8, intermediate=14336, vocab=32000,
                        theta=1000000.0, max_pos=32768, model_type="mixtral", num_local_experts=8,
                        num_experts_per_tok=2, **kw)


# ---------------------------------------------------------------------------------------------
# decoders whose layers differ
# ---------------------------------------------------------------------------------------------
class DictWeights:
    """``Weights`` over tensors that are in memory already."""

    def __new__(cls, tensors: Dict[str, torch.Tensor], device, dtype, bare_names: bool = False):
        from .weights import Weights

        self = Weights([], device, dtype, bare_names=bare_names)

        class _Slice:
            def __init__(self, t):
                self.t = t

            def get_shape(self):
                return tuple(self.t.shape)

            def tensor(self):
                return self.t

            def slice_dim(self, dim, start, stop):
                return self.t.narrow(dim, start, max(0, stop - start)) if self.t.dim() else self.t

        def resolve(name):
            for cand in self._candidates(name):
                if cand in tensors:
                    return None, cand
            raise KeyError(f"weight {name} does not exist")

        self.resolve = resolve
        self._slice = lambda name: _Slice(tensors[resolve(name)[1]])
        return self


def fuzuvik_attention(heads=4, kv_heads=2, dim=32, vdim=16, chunk=48, rot_dims=None, base=10000.0, scaling=None, scale=None,
                      v_mix=True, ff=96) -> dict:
    rot = {"base": base, "dims": dim if rot_dims is None else rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mlp": {"ff": ff, "kind": "dense"} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": rot,
                      "scale": dim ** -0.5 if scale is None else scale, "v_mix": v_mix}}


def fuzuvik_delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, ff=96) -> dict:
    return {"type": "channel_delta", "mlp": {"ff": ff, "kind": "dense"} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def fuzuvik_lightning(heads=3, dim=16, vdim=24, decay=None, ff=96) -> dict:
    decay = decay or [1.0 - 2.0 ** -(1 + 7 * (h + 1) / heads) for h in range(heads)]
    return {"type": "lightning", "mlp": {"ff": ff, "kind": "dense"} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def fuzuvik_config(layers, width=80, vocab=203, eps=1e-5, embed_scale=3.0) -> dict:
    return {"architecture": "Fuzuvik", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "layers": list(layers)}


def fuzuvik_state_dict(cfg: dict, seed: int = 0, dtype=torch.float32, device: str = "cpu",
                       rank: Optional[int] = None) -> Dict[str, torch.Tensor]:
    """Random weights of a Fuzuvik shape.  ``rank``: width of the low-rank decay and gate projections."""
    g = torch.Generator(device=device).manual_seed(seed)
    W, sd = cfg["width"], {}

    def rnd(*shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        return (mean + torch.randn(*shape, generator=g, device=device) * std).to(dtype)

    def uniform(lo, hi, *shape):
        return (lo + (hi - lo) * torch.rand(shape, generator=g, device=device)).to(dtype)

    sd["embed"], sd["head"] = rnd(cfg["vocab"], W, std=0.4), rnd(cfg["vocab"], W)
    sd["final.norm"] = rnd(W, std=0.1, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        mix = p + "mix."
        sd[p + "norm1"] = rnd(W, std=0.1, mean=1.0)
        sd[mix + "o"] = rnd(W, H * dv)
        if layer["type"] == "attention":
            sd.update({mix + "q": rnd(H * d, W), mix + "k": rnd(G * d, W), mix + "v": rnd(G * dv, W),
                       mix + "vmix": uniform(0.2, 0.8)})
        elif layer["type"] == "channel_delta":
            r = rank or max(8, W // 8)
            taps = m["conv"]
            sd.update({mix + "q": rnd(G * d, W), mix + "k": rnd(G * d, W), mix + "v": rnd(H * dv, W), mix + "b": rnd(H, W),
                       mix + "q.conv": rnd(G * d, taps), mix + "k.conv": rnd(G * d, taps), mix + "v.conv": rnd(H * dv, taps),
                       mix + "A_log": uniform(-3.0, 1.0, H), mix + "dt_bias": uniform(-4.0, 0.5, H * d),
                       mix + "norm": rnd(dv, std=0.1, mean=1.0), mix + "a1": rnd(r, W), mix + "a2": rnd(H * d, r),
                       mix + "g1": rnd(r, W), mix + "g2": rnd(H * dv, r)})
        else:
            sd.update({mix + "q": rnd(H * d, W), mix + "k": rnd(H * d, W), mix + "v": rnd(H * dv, W), mix + "g": rnd(H * dv, W),
                       mix + "norm": rnd(H * dv, std=0.1, mean=1.0)})
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            sd.update({p + "norm2": rnd(W, std=0.1, mean=1.0), p + "mlp.up": rnd(ff, W), p + "mlp.down": rnd(W, ff)})
    return sd


def write_checkpoint(path, cfg: dict, sd: Dict[str, torch.Tensor]) -> Path:
    out = Path(path)
    out.mkdir(parents=True, exist_ok=True)
    (out / "config.json").write_text(json.dumps(cfg))
    save_safetensors(sd, out / "model.safetensors")
    return out


def kipedra_attention(heads=4, kv_heads=2, dim=32, vdim=16, window=24, rot_dims=None, base=10000.0, scale=None, conv=4,
                      mlp=None) -> dict:
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window},
                      "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims},
                      "scale": dim ** -0.5 if scale is None else scale}}


def kipedra_delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, mlp=None) -> dict:
    return {"type": "delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def kipedra_dense(ff=96) -> dict:
    return {"kind": "dense", "ff": ff}


def kipedra_moe(ff=40, experts=10, top=3, scale=2.5) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def kipedra_config(layers, width=80, vocab=203, eps=1e-5, residual_mult=0.4, loop=None) -> dict:
    return {"architecture": "Kipedra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": residual_mult,
            "loop": dict(zip(("start", "stop", "times"), loop or (0, len(layers), 1))), "layers": list(layers)}


def kipedra_state_dict(cfg: dict, seed: int = 0, dtype=torch.float32, device: str = "cpu") -> Dict[str, torch.Tensor]:
    """Random weights of a Kipedra shape."""
    g = torch.Generator(device=device).manual_seed(seed)
    W, sd = cfg["width"], {}

    def rnd(*shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        return (mean + torch.randn(*shape, generator=g, device=device) * std).to(dtype)

    def uniform(lo, hi, *shape):
        return (lo + (hi - lo) * torch.rand(shape, generator=g, device=device)).to(dtype)

    sd["embed"], sd["final.norm"] = rnd(cfg["vocab"], W, std=0.5), rnd(W, std=0.2)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        mix, attn = p + "mix.", layer["type"] == "attention"
        sd[p + "norm1"] = rnd(W, std=0.2)
        for n, rows in (("q", (H if attn else G) * d), ("k", G * d), ("v", (G if attn else H) * dv)):
            sd.update({mix + n: rnd(rows, W), mix + n + ".conv": rnd(rows, taps)})
            if attn:
                sd[mix + n + ".b"] = rnd(rows, std=0.3)
        sd[mix + "o"] = rnd(W, H * dv)
        if not attn:
            sd.update({mix + "b": rnd(H, W), mix + "a": rnd(H, W), mix + "g": rnd(H * dv, W), mix + "norm": rnd(dv, std=0.1, mean=1.0),
                       mix + "A_log": uniform(-3.0, 1.0, H), mix + "dt_bias": uniform(-4.0, 0.5, H)})
        if mlp is None:
            continue
        sd[p + "norm2"] = rnd(W, std=0.2)
        if mlp["kind"] == "dense":
            ff = mlp["ff"]
            sd.update({p + "mlp.gate": rnd(ff, W), p + "mlp.up": rnd(ff, W), p + "mlp.down": rnd(W, ff)})
            continue
        ff, E = mlp["expert"]["ff"], mlp["router"]["experts"]
        sd.update({p + "mlp.router": rnd(E, W), p + "mlp.correction": rnd(E, std=0.2)})
        for e in range(E):
            sd.update({f"{p}mlp.e{e}.up": rnd(ff, W), f"{p}mlp.e{e}.down": rnd(W, ff)})
    return sd





def gisilix_attention(heads=4, kv_heads=2, dim=24, vdim=16, coef=0.25, every=20, softcap=9.0, scale=None, kv_from=None,
                      mlp=None) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "q_temp": {"coef": coef, "every": every},
         "softcap": softcap, "scale": dim ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def gisilix_latent(heads=4, dim=24, vdim=20, rank=40, scale=None, mlp=None) -> dict:
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5 if scale is None else scale}}


def gisilix_rotated_latent(heads=4, dim=24, vdim=20, rank=40, rot_dim=8, window=24, base=1000.0, scaling=(4.0, 8.0, 1.0, 128),
                           scale=None, mlp=None) -> dict:
    """``scaling``: (factor, fast, slow, original length)."""
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "fast", "slow", "original"), scaling))
    return {"type": "latent_attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "rot_dim": rot_dim, "mask": {"size": window},
                      "rot": rot, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def gisilix_moe(ff=24, experts=10, top=3, shared=40) -> dict:
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


def gisilix_config(layers, width=80, vocab=203, eps=1e-5) -> dict:
    return {"architecture": "Gisilix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": list(layers)}


def gisilix_state_dict(cfg: dict, seed: int = 0, dtype=torch.float32, device: str = "cpu") -> Dict[str, torch.Tensor]:
    """Random weights of a Gisilix shape."""
    g = torch.Generator(device=device).manual_seed(seed)
    W, sd = cfg["width"], {}

    def rnd(*shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        return (mean + torch.randn(*shape, generator=g, device=device) * std).to(dtype)

    def norm(name, n, bias=True):
        sd[name] = rnd(n, std=0.2, mean=1.0)
        if bias:
            sd[name + ".b"] = rnd(n, std=0.1)

    def feed_forward(p, ff):
        sd.update({p + "gate": rnd(ff, W), p + "up": rnd(ff, W), p + "down": rnd(W, ff)})

    sd["embed"] = rnd(cfg["vocab"], W, std=1.0)
    norm("final.norm", W)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        mix = p + "mix."
        norm(p + "norm1", W)
        sd[mix + "o"] = rnd(W, H * dv)
        if layer["type"] == "attention":
            G = m["kv_heads"]
            sd.update({mix + "q": rnd(H * d, W), mix + "g": rnd(H * dv, W), mix + "sink": rnd(H, std=1.5)})
            norm(mix + "q.norm", H * d, False)
            if m.get("kv_from") is None:
                sd.update({mix + "k": rnd(G * d, W), mix + "v": rnd(G * dv, W)})
                norm(mix + "k.norm", G * d, False)
        else:
            r, rot = m["kv_rank"], m.get("rot_dim", 0)
            sd.update({mix + "q": rnd(H * (d + rot), W), mix + "dkv": rnd(r + rot, W), mix + "uk": rnd(H * d, r), mix + "uv": rnd(H * dv, r)})
            norm(mix + "dkv.norm", r, False)
            if layer["type"] == "latent_attention_2":
                sd[mix + "g"] = rnd(H, W)
        if mlp is None:
            continue
        norm(p + "norm2", W)
        if mlp["kind"] == "dense":
            feed_forward(p + "mlp.", mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        sd.update({p + "mlp.router": rnd(E, W), p + "mlp.router.b": rnd(E, std=0.3)})
        for e in range(E):
            feed_forward(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            feed_forward(p + "mlp.shared.", mlp["shared"]["ff"])
    return sd


# ---- Sobivik: layers normed on both sides, input convolutions, weighted sums over all results ---------------------------
def sobivik_retention(heads=3, dim=24, vdim=20, decay=None, mlp=None) -> dict:
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                                       "decay": decay or [1 - 2.0 ** -(2 + 2 * h) for h in range(heads)]}}


def sobivik_latent(heads=4, dim=24, vdim=20, q_rank=32, kv_rank=40, rot_dim=8, window=24, base=1000.0, scaling=(4.0, 8.0, 1.0, 128),
                   scale=None, mlp=None) -> dict:
    """``scaling``: (factor, fast, slow, original length)."""
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "fast", "slow", "original"), scaling))
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot_dim": rot_dim,
                      "mask": {"size": window}, "rot": rot, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def sobivik_attention(heads=4, kv_heads=2, dim=12, vdim=28, window=20, keep=3, diff=0.3, scale=None, mlp=None) -> dict:
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff,
                      "mask": {"size": window, "keep_first": keep}, "scale": dim ** -0.5 if scale is None else scale}}


def sobivik_config(layers, width=80, vocab=203, eps=1e-5, taps=4, embed_scale=3.0, logit_scale=1.5) -> dict:
    return {"architecture": "Sobivik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": embed_scale}, "logit_scale": logit_scale, "layers": list(layers)}


def sobivik_state_dict(cfg: dict, seed: int = 0, dtype=torch.float32, device: str = "cpu") -> Dict[str, torch.Tensor]:
    """Random weights of a Sobivik shape."""
    g = torch.Generator(device=device).manual_seed(seed)
    W, sd = cfg["width"], {}

    def rnd(*shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        return (mean + torch.randn(shape, generator=g, device=device) * std).to(dtype)

    sd.update({"embed": rnd(cfg["vocab"], W, std=0.4), "head": rnd(cfg["vocab"], W), "final.norm": rnd(std=0.2, mean=1.2)})
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        H, d, dv, mix = m["heads"], m["dim"], m["vdim"], f"l{i}.mix."
        sd.update({p + "norm1": rnd(std=0.2, mean=1.0), p + "norm1b": rnd(std=0.2, mean=0.8), mix + "o": rnd(W, H * dv),
                   p + "canon1": rnd(W, cfg["canon"]["taps"], std=0.3), p + "dwa": rnd(i + 2, std=0.25)})
        sd[p + "dwa"][-1] += 0.8
        if layer["type"] == "retention":
            sd.update({mix + n: rnd(H * w, W) for n, w in (("q", d), ("k", d), ("v", dv), ("g", dv))})
        elif layer["type"] == "latent_attention":
            r, qr, rot = m["kv_rank"], m["q_rank"], m["rot_dim"]
            sd.update({mix + "dq": rnd(qr, W), mix + "dq.norm": rnd(qr, std=0.2, mean=1.0), mix + "uq": rnd(H * (d + rot), qr),
                       mix + "dkv": rnd(r + rot, W), mix + "dkv.norm": rnd(r, std=0.2, mean=1.0), mix + "uk": rnd(H * d, r),
                       mix + "uv": rnd(H * dv, r), mix + "sink": rnd(H, std=1.5), mix + "g": rnd(H * dv, W)})
        else:
            G = m["kv_heads"]
            sd.update({mix + "q": rnd(H * 2 * d, W), mix + "k": rnd(G * 2 * d, W), mix + "v": rnd(G * dv, W), mix + "g": rnd(H, W)})
            sd.update({mix + n: rnd(d, std=0.8 * d ** -0.25) for n in ("lq1", "lk1", "lq2", "lk2")})
        if mlp is not None:
            ff = mlp["ff"]
            sd.update({p + "norm2": rnd(std=0.2, mean=1.0), p + "norm2b": rnd(std=0.2, mean=0.8), p + "mlp.gate": rnd(ff, W),
                       p + "mlp.up": rnd(ff, W), p + "mlp.down": rnd(W, ff)})
    return sd
