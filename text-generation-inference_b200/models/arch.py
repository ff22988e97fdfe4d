"""Architecture descriptions: one generic decoder, many model families.

The reference has one modeling file per family under
``server/text_generation_server/models/custom_modeling/`` (llama ``flash_llama_modeling.py``,
mistral, mixtral, qwen2, gemma/gemma2/gemma3, phi/phi3, cohere, dbrx, gpt2, gptj, neox,
falcon ``flash_rw_modeling.py``, santacoder, starcoder2 ...), all variations of the same
pre-norm decoder.  Here a family is a *declaration* (``Arch``): tensor-name templates plus the
handful of switches in which the families differ; ``models/decoder.py`` interprets it.

``ModelConfig`` is a thin attribute view over ``config.json`` so that no model-specific config
class is needed.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field, replace
from pathlib import Path
from typing import Any, Dict, List, Optional, Tuple


def _fuzuvik_config(d: Dict[str, Any]) -> Dict[str, Any]:
    """Fuzuvik checkpoints describe every layer on its own (``layers``: mixer type, its sizes, its feed-forward) and use
    their own key names; brought here to the names the rest of the package reads, with the layers as ``MixerSpec``s."""
    out = dict(d)
    layers = d["layers"]
    specs = []
    for i, layer in enumerate(layers):
        m, mlp = layer["mixer"], layer.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        ff = 0 if mlp is None else int(mlp["ff"])
        sizes = dict(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=int(m["dim"]),
                     vdim=int(m["vdim"]), ff=ff)
        if layer["type"] == "attention":
            rot = m.get("rot") or {}
            sc = rot.get("scaling")
            specs.append(MixerSpec(
                "attention", **sizes, scale=float(m["scale"]), chunk=int((m.get("mask") or {}).get("size") or 0), sink=True,
                qk_unit_rms=True, v_mix=bool(m.get("v_mix")), rot_dims=int(rot.get("dims") or 0),
                rot_base=float(rot.get("base") or 10000.0),
                rot_scaling=None if not sc else (float(sc["factor"]), float(sc["low"]), float(sc["high"]), float(sc["original"]))))
        elif layer["type"] == "channel_delta":
            specs.append(MixerSpec("delta", **sizes, short_conv=True))
        elif layer["type"] == "lightning":
            specs.append(MixerSpec("decay", **sizes, decay=tuple(float(x) for x in m["decay"])))
        else:
            raise NotImplementedError(f"layer {i}: mixer {layer['type']!r}")
    attn = [s for s in specs if s.kind == "attention"]
    out.update(model_type="fuzuvik", hidden_size=int(d["width"]), vocab_size=int(d["vocab"]), num_hidden_layers=len(layers),
               num_attention_heads=max(s.heads for s in (attn or specs)), rms_norm_eps=float(d["norm"]["eps"]),
               embedding_multiplier=float((d.get("embedding") or {}).get("scale", 1.0)), mixers=specs,
               # rotary positions are unbounded by design: the table length is a deployment choice
               max_position_embeddings=int(d.get("max_position_embeddings") or 131072))
    return out


def _layer_order(count: int, loop: Optional[Dict[str, Any]]) -> List[int]:
    """Layers in the order they run: ``loop`` repeats layers ``start .. stop - 1`` ``times`` times in a row."""
    if not loop:
        return list(range(count))
    lo, hi, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= lo <= hi <= count or times < 1:
        raise ValueError(f"a loop over layers {lo} .. {hi - 1}, {times} times, does not fit {count} layers")
    return list(range(lo)) + list(range(lo, hi)) * times + list(range(hi, count))


def _kipedra_config(d: Dict[str, Any]) -> Dict[str, Any]:
    """Kipedra checkpoints: layers described one by one as in Fuzuvik's, mixer and feed-forward side by side, layers that
    may run several times."""
    out = dict(d)
    layers = d["layers"]
    specs = []
    for i, layer in enumerate(layers):
        m, mlp = layer["mixer"], layer.get("mlp")
        ff, moe = 0, None
        if mlp is not None and mlp["kind"] == "dense":
            ff = int(mlp["ff"])
        elif mlp is not None and mlp["kind"] == "moe":
            r = mlp["router"]
            moe = ExpertSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), scale=float(r["scale"]),
                             act="relu2")
        elif mlp is not None:
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        sizes = dict(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=int(m["dim"]),
                     vdim=int(m["vdim"]), ff=ff, moe=moe)
        if layer["type"] == "attention":
            rot = m.get("rot") or {}
            specs.append(MixerSpec(
                "attention", **sizes, scale=float(m["scale"]), window=int((m.get("mask") or {}).get("size") or 0),
                short_conv=bool(m.get("conv")), qkv_bias=True, rot_dims=int(rot.get("dims") or 0), rot_base=float(rot.get("base") or 10000.0),
                rot_interleaved=True))
        elif layer["type"] == "delta":
            specs.append(MixerSpec("delta", **sizes, short_conv=True, head_decay=True, gate_act="silu"))
        else:
            raise NotImplementedError(f"layer {i}: mixer {layer['type']!r}")
    attn = [s for s in specs if s.kind == "attention"]
    out.update(model_type="kipedra", hidden_size=int(d["width"]), vocab_size=int(d["vocab"]), num_hidden_layers=len(layers),
               num_attention_heads=max(s.heads for s in (attn or specs)), rms_norm_eps=float(d["norm"]["eps"]),
               residual_multiplier=float(d.get("residual_mult", 1.0)), mixers=specs,
               layer_order=_layer_order(len(layers), d.get("loop")), tie_word_embeddings=True,
               # rotary positions are unbounded by design: the table length is a deployment choice
               max_position_embeddings=int(d.get("max_position_embeddings") or 131072))
    return out


def _gisilix_config(d: Dict[str, Any]) -> Dict[str, Any]:
    """Gisilix checkpoints: layers described one by one as in Fuzuvik's; attention over latents, attention with learned sinks
    whose keys and values other layers may share, softmax-routed gated experts beside a shared one."""
    out = dict(d)
    layers = d["layers"]
    specs = []
    for i, layer in enumerate(layers):
        m, mlp = layer["mixer"], layer.get("mlp")
        ff, moe = 0, None
        if mlp is not None and mlp["kind"] == "dense":
            ff = int(mlp["ff"])
        elif mlp is not None and mlp["kind"] == "moe":
            r = mlp["router"]
            moe = ExpertSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), act="silu", gated=True,
                             router="softmax", shared_ff=int((mlp.get("shared") or {}).get("ff") or 0))
        elif mlp is not None:
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        sizes = dict(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=int(m["dim"]),
                     vdim=int(m["vdim"]), ff=ff, moe=moe, scale=float(m["scale"]),
                     window=int((m.get("mask") or {}).get("size") or 0))
        if layer["type"] == "attention":
            temp, src = m.get("q_temp"), m.get("kv_from")
            specs.append(MixerSpec(
                "attention", **sizes, row_norm=True, softcap=float(m.get("softcap") or 0.0), learned_sink=True,
                q_temp=None if not temp else (float(temp["coef"]), int(temp["every"])), out_gate="element",
                kv_from=None if src is None else int(src)))
        elif layer["type"] in ("latent_attention", "latent_attention_2"):
            rotated = layer["type"] == "latent_attention_2"
            rot = (m.get("rot") or {}) if rotated else {}
            sc = rot.get("scaling")
            specs.append(MixerSpec(
                "latent", **{**sizes, "kv_heads": 1}, kv_rank=int(m["kv_rank"]), rot_dims=int(m.get("rot_dim") or 0) if rotated else 0,
                rot_base=float(rot.get("base") or 10000.0), rot_interleaved=True,
                rot_yarn=None if not sc else tuple(float(sc[k]) for k in ("factor", "fast", "slow", "original")),
                out_gate="head" if rotated else ""))
        else:
            raise NotImplementedError(f"layer {i}: mixer {layer['type']!r}")
    for i, s in enumerate(specs):
        if s.kv_from is not None:
            src = specs[s.kv_from] if 0 <= s.kv_from < i else None
            if src is None or src.kind != "attention" or src.kv_from is not None or (src.kv_heads, src.dim, src.vdim) != (s.kv_heads, s.dim, s.vdim):
                raise ValueError(f"layer {i} cannot use the keys and values of layer {s.kv_from}")
    out.update(model_type="gisilix", hidden_size=int(d["width"]), vocab_size=int(d["vocab"]), num_hidden_layers=len(layers),
               num_attention_heads=max(s.heads for s in specs), rms_norm_eps=float(d["norm"]["eps"]), mixers=specs,
               tie_word_embeddings=True,
               # rotary positions are unbounded by design: the table length is a deployment choice
               max_position_embeddings=int(d.get("max_position_embeddings") or 131072))
    return out


def _sobivik_config(d: Dict[str, Any]) -> Dict[str, Any]:
    """Sobivik checkpoints: layers described one by one as in Fuzuvik's; retention, latent attention with a latent for the
    queries too, differential attention; norms of one number around both halves of a layer, a convolution on what a mixer
    reads, and a weighted sum over the results of all layers so far."""
    out = dict(d)
    layers = d["layers"]
    taps = int((d.get("canon") or {}).get("taps") or 0)
    specs = []
    for i, layer in enumerate(layers):
        m, mlp = layer["mixer"], layer.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        mask = m.get("mask") or {}
        sizes = dict(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads") or m["heads"]), dim=int(m["dim"]),
                     vdim=int(m["vdim"]), ff=0 if mlp is None else int(mlp["ff"]), input_conv=taps)
        if layer["type"] == "retention":
            specs.append(MixerSpec("decay", **sizes, decay=tuple(float(x) for x in m["decay"]), qkv_act="",
                                   k_scale=float(m["dim"]) ** -0.5, head_norm=True, gate_act="silu"))
        elif layer["type"] == "latent_attention":
            rot = m["rot"]
            sc = rot.get("scaling")
            if int(rot["dims"]) != int(m["rot_dim"]):
                raise NotImplementedError(f"layer {i}: {rot['dims']} of {m['rot_dim']} key dimensions rotated")
            specs.append(MixerSpec(
                "latent", **{**sizes, "kv_heads": 1}, scale=float(m["scale"]), window=int(mask.get("size") or 0),
                kv_rank=int(m["kv_rank"]), q_rank=int(m["q_rank"]), rot_dims=int(m["rot_dim"]), rot_base=float(rot["base"]),
                rot_yarn=None if not sc else tuple(float(sc[k]) for k in ("factor", "fast", "slow", "original")),
                learned_sink=True, out_gate="element"))
        elif layer["type"] == "attention":
            specs.append(MixerSpec(
                "attention", **sizes, scale=float(m["scale"]), window=int(mask.get("size") or 0),
                keep_first=int(mask.get("keep_first") or 0), diff=float(m["diff"]), out_gate="head"))
        else:
            raise NotImplementedError(f"layer {i}: mixer {layer['type']!r}")
    out.update(model_type="sobivik", hidden_size=int(d["width"]), vocab_size=int(d["vocab"]), num_hidden_layers=len(layers),
               num_attention_heads=max(s.heads for s in specs), rms_norm_eps=float(d["norm"]["eps"]),
               embedding_multiplier=float((d.get("embedding") or {}).get("scale", 1.0)),
               logit_scale=float(d.get("logit_scale", 1.0)), mixers=specs,
               # rotary positions are unbounded by design: the table length is a deployment choice
               max_position_embeddings=int(d.get("max_position_embeddings") or 131072))
    return out


# ``architecture`` of a config.json without ``model_type`` -> function that brings it to the common names
CONFIG_READERS = {"Fuzuvik": _fuzuvik_config, "Kipedra": _kipedra_config, "Gisilix": _gisilix_config,
                  "Sobivik": _sobivik_config}


class ModelConfig:
    """Attribute access to ``config.json`` with ``get``-style defaults; unknown attributes are ``None``."""

    def __init__(self, data: Dict[str, Any]):
        reader = CONFIG_READERS.get(data.get("architecture")) if "model_type" not in data else None
        object.__setattr__(self, "_d", reader(data) if reader else dict(data))

    @classmethod
    def from_path(cls, path) -> "ModelConfig":
        p = Path(path)
        if p.is_dir():
            p = p / "config.json"
        return cls(json.loads(p.read_text()))

    def __getattr__(self, k):
        if k.startswith("__"):
            raise AttributeError(k)
        return self._d.get(k)

    def __setattr__(self, k, v):
        self._d[k] = v

    def get(self, k, default=None):
        v = self._d.get(k)
        return default if v is None else v

    def to_dict(self):
        return dict(self._d)

    def text_config(self) -> "ModelConfig":
        """Language-model part of a multimodal config."""
        t = self._d.get("text_config")
        if isinstance(t, dict):
            merged = dict(t)
            merged.setdefault("quantization_config", self._d.get("quantization_config"))
            return ModelConfig(merged)
        return self


@dataclass(frozen=True)
class ExpertSpec:
    """Routed feed-forward of one layer: experts ``down(act(up(h)))``, or ``down(act(gate(h)) * up(h))`` when ``gated``.

    ``router="sigmoid"``: chosen by the sigmoid of their router logits plus a stored correction, weighted by the sigmoids
    alone, which are brought to the sum ``scale``.  ``router="softmax"``: chosen by their router logits, stored bias included,
    weighted by the softmax over the chosen logits."""

    experts: int
    top: int                                 # experts per token
    ff: int                                  # width of an expert
    scale: float = 1.0
    act: str = "relu2"
    gated: bool = False
    router: str = "sigmoid"
    shared_ff: int = 0                       # width of a feed-forward that every token runs beside its experts, 0: none


@dataclass(frozen=True)
class MixerSpec:
    """Token mixer and feed-forward of one layer of a decoder whose layers differ (``models/mixers.py``)."""

    kind: str                                # "attention" | "latent" (attention over a latent that all heads share) |
                                             # "delta" (gated delta rule) | "decay" (fixed decay per head)
    heads: int
    kv_heads: int                            # attention: key/value heads; delta: query/key heads
    dim: int                                 # query / key size of a head
    vdim: int                                # value size of a head
    ff: int = 0                              # width of a dense feed-forward, 0: the layer has none
    moe: Optional[ExpertSpec] = None         # routed experts in its place
    short_conv: bool = False                 # causal convolution over time on every channel of q, k and v
    input_conv: int = 0                      # taps of a causal convolution over time added to what the mixer reads
    # attention, latent
    scale: float = 1.0
    window: int = 0                          # > 0: the token itself and the window - 1 tokens before it
    keep_first: int = 0                      # first tokens of a sequence that stay visible past the window
    chunk: int = 0                           # > 0: keys of the query's own chunk of this many positions
    sink: bool = False                       # one more key of score 0, without a value, in the softmax
    learned_sink: bool = False               # the same with a stored score per head
    softcap: float = 0.0                     # > 0: scores become softcap * tanh(score / softcap)
    qk_unit_rms: bool = False                # q and k over their root mean square, after the rotation
    row_norm: bool = False                   # q and k normed over all heads at once, with weights (no rotation)
    q_temp: Optional[Tuple[float, int]] = None    # (coef, every): q times 1 + coef * ln(floor((p + 1) / every) + 1)
    out_gate: str = ""                       # output times the sigmoid of a projection: "element" | "head" (one per head)
    kv_from: Optional[int] = None            # layer whose keys and values this one reads
    diff: Optional[float] = None             # two maps per head over the same values: the first minus lambda times the
                                             # second, normed per head, times 1 - diff (lambda: learned part + diff)
    kv_rank: int = 0                         # latent: its size
    q_rank: int = 0                          # latent: > 0: queries come from a normed latent of this size
    v_mix: bool = False                      # values mixed with those of the first such layer
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_scaling: Optional[Tuple[float, float, float, float]] = None    # (factor, low, high, original length)
    rot_yarn: Optional[Tuple[float, float, float, float]] = None       # (factor, fast, slow, original length)
    rot_interleaved: bool = False            # pairs 2i, 2i + 1 (False: i, i + rot_dims / 2)
    qkv_bias: bool = False
    # delta
    head_decay: bool = False                 # one decay per head, full-rank decay and gate projections (False: one per
                                             # head and key channel, low-rank projections)
    gate_act: str = "sigmoid"                # of the output gate
    # decay
    decay: Tuple[float, ...] = ()
    qkv_act: str = "silu"                    # of q, k and v, "": none
    k_scale: float = 1.0                     # factor of k
    head_norm: bool = False                  # weightless norm per head (False: one weighted norm over all heads)

    @property
    def paged(self) -> bool:
        """Keeps something of every token: keys and values, or what they are made from."""
        return self.kind in ("attention", "latent")

    @property
    def recurrent(self) -> bool:
        """Keeps a state per sequence that every token advances."""
        return not self.paged or self.short_conv or self.input_conv > 0

    @property
    def feed_forward(self) -> bool:
        return self.ff > 0 or self.moe is not None


@dataclass(frozen=True)
class Arch:
    # ---- tensor names ------------------------------------------------------------------------
    embed: str = "model.embed_tokens"
    pos_embed: Optional[str] = None          # learned absolute positions (gpt2, opt)
    pos_offset: int = 0                      # opt adds 2 to positions
    embed_norm: Optional[str] = None         # bloom word_embeddings_layernorm
    layer: str = "model.layers.{i}"
    norm1: str = "input_layernorm"
    norm2: Optional[str] = "post_attention_layernorm"
    post_attn_norm: Optional[str] = None     # gemma2/3: norm on the attention output
    post_mlp_norm: Optional[str] = None      # gemma2/3: norm on the MLP output
    final_norm: str = "model.norm"
    lm_head: str = "lm_head"
    q: str = "self_attn.q_proj"
    k: str = "self_attn.k_proj"
    v: str = "self_attn.v_proj"
    qkv: Optional[str] = None                # fused projection name, if the checkpoint fuses q,k,v
    qkv_layout: str = "blocked"              # "blocked" [q|k|v], "interleaved" per-head [q,k,v] (neox, bloom), "falcon"
    o: str = "self_attn.o_proj"
    q_norm: Optional[str] = None
    k_norm: Optional[str] = None
    gate: Optional[str] = "mlp.gate_proj"
    up: str = "mlp.up_proj"
    gate_up: Optional[str] = None            # fused gate+up name
    down: str = "mlp.down_proj"
    conv1d_weights: bool = False             # gpt2 stores linear weights transposed
    # ---- behaviour ---------------------------------------------------------------------------
    norm: str = "rms"                        # "rms" | "layer"
    norm_unit_offset: bool = False           # gemma: weight + 1
    norm_bias: bool = True                   # layer norm with bias
    qkv_bias: bool = False
    o_bias: bool = False
    mlp_bias: bool = False
    act: Optional[str] = None                # None: from config.hidden_act
    gated_mlp: bool = True
    parallel_residual: bool = False
    parallel_shared_norm: bool = True        # parallel blocks: one norm feeds attention and MLP
    rope: bool = True
    rope_neox: bool = True
    alibi: bool = False
    embed_scale_sqrt_hidden: bool = False    # gemma
    qk_norm_kind: str = "rms"                # "rms" per-head over head_dim | "layer" (cohere)
    # ---- mixture of experts ------------------------------------------------------------------
    moe: bool = False
    moe_router: str = "block_sparse_moe.gate"
    moe_expert: str = "block_sparse_moe.experts.{e}"
    moe_gate: str = "w1"
    moe_up: str = "w3"
    moe_down: str = "w2"
    moe_fused: bool = False                  # dbrx: experts stored stacked
    moe_shared: Optional[str] = None         # shared expert MLP prefix (qwen2_moe, deepseek)
    mla: bool = False                        # DeepSeek multi-head latent attention (models/deepseek.py)
    moe_shared_gate: Optional[str] = None
    moe_renormalize: bool = True
    moe_correction: Optional[str] = None     # correction of the choice scores, or bias of the logits (layers with an `ExpertSpec`)
    # ---- layers that differ (config "mixers") ---------------------------------------------------
    mix: Optional[str] = None                # tensor prefix of a layer's mixer
    input_conv: Optional[str] = None         # layers with `MixerSpec.input_conv`: its tensor
    depth_average: Optional[str] = None      # weights of the embedding output and of all layers' results so far, whose sum goes on
    residual_fp32: bool = False              # the residual stream is kept in 32 bits
    bare_names: bool = False                 # tensors are named without the ".weight" suffix, biases end in ".b"


_LLAMA = Arch()

ARCHS: Dict[str, Arch] = {
    "llama": _LLAMA,
    "mistral": _LLAMA,
    "baichuan": replace(_LLAMA, qkv="self_attn.W_pack"),
    "granite": _LLAMA,
    "qwen2": replace(_LLAMA, qkv_bias=True),
    "qwen3": replace(_LLAMA, q_norm="self_attn.q_norm", k_norm="self_attn.k_norm"),
    "phi3": replace(_LLAMA, qkv="self_attn.qkv_proj", gate=None, gate_up="mlp.gate_up_proj"),
    "gemma": replace(_LLAMA, norm_unit_offset=True, embed_scale_sqrt_hidden=True),
    "gemma2": replace(_LLAMA, norm_unit_offset=True, embed_scale_sqrt_hidden=True,
                      norm2="pre_feedforward_layernorm", post_attn_norm="post_attention_layernorm",
                      post_mlp_norm="post_feedforward_layernorm"),
    "gemma3_text": replace(_LLAMA, norm_unit_offset=True, embed_scale_sqrt_hidden=True,
                           norm2="pre_feedforward_layernorm", post_attn_norm="post_attention_layernorm",
                           post_mlp_norm="post_feedforward_layernorm",
                           q_norm="self_attn.q_norm", k_norm="self_attn.k_norm"),
    "starcoder2": replace(_LLAMA, norm="layer", qkv_bias=True, o_bias=True, mlp_bias=True, gated_mlp=False,
                          gate=None, up="mlp.c_fc", down="mlp.c_proj"),
    "cohere": replace(_LLAMA, norm="layer", norm_bias=False, norm2=None, parallel_residual=True, rope_neox=False,
                      q_norm="self_attn.q_norm", k_norm="self_attn.k_norm", qk_norm_kind="layer"),
    "mixtral": replace(_LLAMA, moe=True),
    "phimoe": replace(_LLAMA, moe=True, norm="layer", qkv_bias=True, o_bias=True),
    "qwen2_moe": replace(_LLAMA, qkv_bias=True, moe=True, moe_router="mlp.gate", moe_expert="mlp.experts.{e}",
                         moe_gate="gate_proj", moe_up="up_proj", moe_down="down_proj",
                         moe_shared="mlp.shared_expert", moe_shared_gate="mlp.shared_expert_gate",
                         moe_renormalize=False),
    "qwen3_moe": replace(_LLAMA, q_norm="self_attn.q_norm", k_norm="self_attn.k_norm", moe=True,
                         moe_router="mlp.gate", moe_expert="mlp.experts.{e}", moe_gate="gate_proj",
                         moe_up="up_proj", moe_down="down_proj"),
    "gpt2": Arch(embed="wte", pos_embed="wpe", layer="h.{i}", norm1="ln_1", norm2="ln_2", final_norm="ln_f",
                 lm_head="lm_head", qkv="attn.c_attn", o="attn.c_proj", gate=None, up="mlp.c_fc",
                 down="mlp.c_proj", conv1d_weights=True, norm="layer", qkv_bias=True, o_bias=True,
                 mlp_bias=True, gated_mlp=False, rope=False),
    "gpt_bigcode": Arch(embed="transformer.wte", pos_embed="transformer.wpe", layer="transformer.h.{i}",
                        norm1="ln_1", norm2="ln_2", final_norm="transformer.ln_f", lm_head="lm_head",
                        qkv="attn.c_attn", o="attn.c_proj", gate=None, up="mlp.c_fc", down="mlp.c_proj",
                        norm="layer", qkv_bias=True, o_bias=True, mlp_bias=True, gated_mlp=False, rope=False),
    "gptj": Arch(embed="transformer.wte", layer="transformer.h.{i}", norm1="ln_1", norm2=None,
                 final_norm="transformer.ln_f", q="attn.q_proj", k="attn.k_proj", v="attn.v_proj",
                 o="attn.out_proj", gate=None, up="mlp.fc_in", down="mlp.fc_out", norm="layer",
                 mlp_bias=True, gated_mlp=False, parallel_residual=True, rope_neox=False),
    "gpt_neox": Arch(embed="gpt_neox.embed_in", layer="gpt_neox.layers.{i}", norm1="input_layernorm",
                     norm2="post_attention_layernorm", final_norm="gpt_neox.final_layer_norm",
                     lm_head="embed_out", qkv="attention.query_key_value", qkv_layout="interleaved",
                     o="attention.dense", gate=None, up="mlp.dense_h_to_4h", down="mlp.dense_4h_to_h",
                     norm="layer", qkv_bias=True, o_bias=True, mlp_bias=True, gated_mlp=False,
                     parallel_residual=True, parallel_shared_norm=False),
    "phi": Arch(layer="model.layers.{i}", norm1="input_layernorm", norm2=None, final_norm="model.final_layernorm",
                o="self_attn.dense", gate=None, up="mlp.fc1", down="mlp.fc2", norm="layer", qkv_bias=True,
                o_bias=True, mlp_bias=True, gated_mlp=False, parallel_residual=True),
    "falcon": Arch(embed="transformer.word_embeddings", layer="transformer.h.{i}", norm1="input_layernorm",
                   norm2=None, final_norm="transformer.ln_f", qkv="self_attention.query_key_value",
                   qkv_layout="falcon", o="self_attention.dense", gate=None, up="mlp.dense_h_to_4h",
                   down="mlp.dense_4h_to_h", norm="layer", gated_mlp=False, parallel_residual=True),
    "bloom": Arch(embed="word_embeddings", embed_norm="word_embeddings_layernorm", layer="h.{i}",
                  norm1="input_layernorm", norm2="post_attention_layernorm", final_norm="ln_f",
                  lm_head="lm_head", qkv="self_attention.query_key_value", qkv_layout="interleaved",
                  o="self_attention.dense", gate=None, up="mlp.dense_h_to_4h", down="mlp.dense_4h_to_h",
                  norm="layer", qkv_bias=True, o_bias=True, mlp_bias=True, gated_mlp=False, rope=False, alibi=True),
    "mpt": Arch(embed="transformer.wte", layer="transformer.blocks.{i}", norm1="norm_1", norm2="norm_2",
                final_norm="transformer.norm_f", qkv="attn.Wqkv", o="attn.out_proj", gate=None,
                up="ffn.up_proj", down="ffn.down_proj", norm="layer", norm_bias=False, gated_mlp=False,
                rope=False, alibi=True),
    "opt": Arch(embed="model.decoder.embed_tokens", pos_embed="model.decoder.embed_positions", pos_offset=2,
                layer="model.decoder.layers.{i}", norm1="self_attn_layer_norm", norm2="final_layer_norm",
                final_norm="model.decoder.final_layer_norm", o="self_attn.out_proj", gate=None, up="fc1",
                down="fc2", norm="layer", qkv_bias=True, o_bias=True, mlp_bias=True, gated_mlp=False, rope=False),
    "dbrx": Arch(embed="transformer.wte", layer="transformer.blocks.{i}", norm1="norm_attn_norm.norm_1",
                 norm2="norm_attn_norm.norm_2", final_norm="transformer.norm_f",
                 qkv="norm_attn_norm.attn.Wqkv", o="norm_attn_norm.attn.out_proj", norm="layer", norm_bias=False,
                 moe=True, moe_router="ffn.router.layer", moe_expert="ffn.experts.mlp", moe_fused=True,
                 moe_gate="w1", moe_up="v1", moe_down="w2"),
}
ARCHS["RefinedWeb"] = ARCHS["RefinedWebModel"] = ARCHS["falcon"]
ARCHS["deepseek_v2"] = ARCHS["deepseek_v3"] = replace(
    _LLAMA, rope_neox=False, mla=True, moe=True, moe_router="mlp.gate", moe_expert="mlp.experts.{e}",
    moe_gate="gate_proj", moe_up="up_proj", moe_down="down_proj", moe_shared="mlp.shared_experts")
# decoder whose layers mix tokens in different ways; names inside a mixer are in models/mixers.py
ARCHS["fuzuvik"] = Arch(embed="embed", layer="l{i}", norm1="norm1", norm2="norm2", final_norm="final.norm", lm_head="head",
                        mix="mix", gate=None, up="mlp.up", down="mlp.down", gated_mlp=False, act="gelu", rope=False,
                        residual_fp32=True, bare_names=True)
ARCHS["kipedra"] = Arch(embed="embed", layer="l{i}", norm1="norm1", norm2="norm2", final_norm="final.norm", lm_head="head",
                        mix="mix", gate="mlp.gate", up="mlp.up", down="mlp.down", act="gelu_tanh", rope=False,
                        norm_unit_offset=True, parallel_residual=True, parallel_shared_norm=False, residual_fp32=True,
                        bare_names=True, moe_router="mlp.router", moe_expert="mlp.e{e}", moe_up="up", moe_down="down",
                        moe_correction="mlp.correction")
ARCHS["gisilix"] = Arch(embed="embed", layer="l{i}", norm1="norm1", norm2="norm2", final_norm="final.norm", lm_head="head",
                        mix="mix", gate="mlp.gate", up="mlp.up", down="mlp.down", act="silu", rope=False, norm="layer",
                        residual_fp32=True, bare_names=True, moe_router="mlp.router", moe_expert="mlp.e{e}", moe_gate="gate",
                        moe_up="up", moe_down="down", moe_correction="mlp.router.b", moe_shared="mlp.shared")
ARCHS["sobivik"] = Arch(embed="embed", layer="l{i}", norm1="norm1", norm2="norm2", post_attn_norm="norm1b", post_mlp_norm="norm2b",
                        final_norm="final.norm", lm_head="head", mix="mix", input_conv="canon1", depth_average="dwa",
                        gate="mlp.gate", up="mlp.up", down="mlp.down", act="silu", rope=False, residual_fp32=True, bare_names=True)
ARCHS["gemma3"] = ARCHS["gemma3_text"]
ARCHS["phi-msft"] = ARCHS["phi"]
ARCHS["qwen2_vl_text"] = ARCHS["qwen2_5_vl_text"] = ARCHS["qwen2"]   # language models of Qwen2-VL / Qwen2.5-VL


def arch_for(model_type: str) -> Arch:
    if model_type not in ARCHS:
        raise NotImplementedError(f"model type {model_type} has no architecture description")
    return ARCHS[model_type]


@dataclass
class ModelDims:
    """Numbers derived from the config, after tensor-parallel division."""

    hidden: int
    num_layers: int
    num_heads: int          # per rank
    num_kv_heads: int       # per rank
    head_dim: int
    intermediate: int
    vocab: int
    eps: float
    rope_theta: float
    rot_dim: int
    max_positions: int
    act: str
    softmax_scale: float
    windows: List[int]      # per layer, -1 = full attention
    attn_softcap: float
    logit_softcap: float
    logit_scale: float
    embed_scale: float
    residual_scale: float
    num_experts: int = 0
    top_k: int = 0
    total_heads: int = 0
    total_kv_heads: int = 0
    mixers: Optional[List[MixerSpec]] = None    # per layer, for decoders whose layers differ
    layer_order: Optional[List[int]] = None     # layers in the order they run (None: each once)
    attn_head_dim: int = 0      # head dimension seen by the attention kernels and the KV cache: head_dim padded to 64/128/256


def derive_dims(cfg: ModelConfig, arch: Arch, world: int) -> ModelDims:
    hidden = cfg.get("hidden_size", cfg.get("n_embd", cfg.get("d_model")))
    layers = cfg.get("num_hidden_layers", cfg.get("n_layer", cfg.get("n_layers")))
    heads = cfg.get("num_attention_heads", cfg.get("n_head", cfg.get("n_heads")))
    head_dim = cfg.get("head_dim", hidden // heads)
    kv = cfg.get("num_key_value_heads")
    if arch.mla:
        # latent attention is expanded to ordinary heads of a padded dimension (models/deepseek.py)
        head_dim, kv = 256, heads
    if kv is None and cfg.get("new_decoder_architecture") and cfg.get("num_kv_heads") is not None:
        kv = cfg.get("num_kv_heads")     # Falcon-40B style: grouped KV heads, `multi_query` is ignored
    if kv is None:
        if cfg.get("attention_head_type") == "multiquery":        # the first SantaCoder checkpoints
            kv = 1
        elif cfg.get("multi_query") or (cfg.model_type in ("falcon", "RefinedWebModel", "RefinedWeb")
                                      and cfg.get("multi_query", True) and not cfg.get("new_decoder_architecture")):
            kv = 1
        elif cfg.get("n_head_kv") is not None or cfg.get("num_kv_heads") is not None:
            kv = cfg.get("n_head_kv", cfg.get("num_kv_heads"))
        elif isinstance(cfg.get("attn_config"), dict) and cfg.attn_config.get("kv_n_heads"):
            kv = cfg.attn_config["kv_n_heads"]
        else:
            kv = heads
    if heads % world != 0:
        raise ValueError(f"`num_heads` must be divisible by `num_shards` (got `num_heads`: {heads} "
                         f"and `num_shards`: {world}")
    # MQA / few KV heads: replicate KV heads when there are fewer than ranks.
    kv_local = kv // world if kv >= world else 1
    if kv >= world and kv % world != 0:
        raise ValueError(f"`num_key_value_heads` ({kv}) must be divisible by `num_shards` ({world})")
    inter = cfg.get("intermediate_size", cfg.get("n_inner", cfg.get("ffn_hidden_size")))
    if inter is None:
        ffn = cfg.get("ffn_config") if isinstance(cfg.get("ffn_config"), dict) else {}
        inter = ffn.get("ffn_hidden_size", 4 * hidden)
    eps = cfg.get("rms_norm_eps", cfg.get("layer_norm_eps", cfg.get("layer_norm_epsilon", cfg.get("norm_epsilon", 1e-5))))
    act = arch.act or cfg.get("hidden_act", cfg.get("hidden_activation", cfg.get("activation_function", "gelu")))
    rope_params = cfg.get("rope_parameters") if isinstance(cfg.get("rope_parameters"), dict) else {}
    full = rope_params.get("full_attention") if isinstance(rope_params.get("full_attention"), dict) else {}
    attn_cfg = cfg.get("attn_config") if isinstance(cfg.get("attn_config"), dict) else {}
    theta = 10000.0
    for cand in (cfg.get("rope_theta"), rope_params.get("rope_theta"), full.get("rope_theta"), attn_cfg.get("rope_theta"),
                 cfg.get("rotary_emb_base")):
        if cand is not None:
            theta = float(cand)
            break
    partial = cfg.get("partial_rotary_factor", cfg.get("rotary_pct", 1.0))
    rot = cfg.get("rotary_dim")
    if arch.mla:
        rot = int(cfg.qk_rope_head_dim)
    if rot is None:
        rot = int(head_dim * partial)
    rot_dim = rot if arch.rope else 0
    max_pos = cfg.get("max_position_embeddings", cfg.get("n_positions", cfg.get("max_seq_len", 2048)))
    scalar = cfg.get("query_pre_attn_scalar")
    scale = (scalar ** -0.5) if scalar else head_dim ** -0.5
    if cfg.get("attention_multiplier"):
        scale = float(cfg.attention_multiplier)
    window = cfg.get("sliding_window")
    windows = [-1] * layers
    if window and cfg.get("use_sliding_window", True):
        if cfg.model_type == "gemma2":
            windows = [window if i % 2 == 0 else -1 for i in range(layers)]
        elif cfg.model_type in ("gemma3", "gemma3_text"):
            pat = cfg.get("sliding_window_pattern", 6)
            lt = cfg.get("layer_types")
            windows = [(window if (lt[i] == "sliding_attention" if lt else (i + 1) % pat != 0) else -1)
                       for i in range(layers)]
        elif cfg.model_type == "qwen2" and cfg.get("max_window_layers") is not None:
            windows = [window if i >= cfg.max_window_layers else -1 for i in range(layers)]
        else:
            windows = [window] * layers
    mixers = cfg.get("mixers")
    if mixers:
        # sizes are per layer; the scalars below describe the widest attention layer and are informative only
        if world != 1:
            raise NotImplementedError(f"{cfg.model_type} is served on one GPU: its mixers are not sharded")
        head_dim = 64
    ne = cfg.get("num_local_experts", cfg.get("num_experts", cfg.get("n_routed_experts", 0))) or 0
    tk = cfg.get("num_experts_per_tok", cfg.get("moe_top_k", 0)) or 0
    if isinstance(cfg.get("ffn_config"), dict):
        ne = cfg.ffn_config.get("moe_num_experts", ne)
        tk = cfg.ffn_config.get("moe_top_k", tk)
    if arch.moe and cfg.get("moe_intermediate_size"):
        inter = cfg.moe_intermediate_size
    attn_dim = next((d for d in (64, 128, 256) if d >= head_dim), None)
    if attn_dim is None:
        raise ValueError(f"head dimension {head_dim} is larger than the attention kernels support (256)")
    return ModelDims(
        attn_head_dim=attn_dim,
        hidden=hidden, num_layers=layers, num_heads=heads // world, num_kv_heads=kv_local, head_dim=head_dim,
        intermediate=inter, vocab=cfg.get("vocab_size"), eps=float(eps), rope_theta=theta, rot_dim=rot_dim,
        max_positions=max_pos, act=act, softmax_scale=scale, windows=windows,
        attn_softcap=float(cfg.get("attn_logit_softcapping", 0.0) or 0.0),
        logit_softcap=float(cfg.get("final_logit_softcapping", 0.0) or 0.0),
        logit_scale=float(cfg.get("logit_scale", 1.0) or 1.0) / float(cfg.get("logits_scaling", 1.0) or 1.0),
        embed_scale=(math.sqrt(hidden) if arch.embed_scale_sqrt_hidden else float(cfg.get("embedding_multiplier", 1.0) or 1.0)),
        residual_scale=float(cfg.get("residual_multiplier", 1.0) or 1.0),
        num_experts=ne, top_k=tk, total_heads=heads, total_kv_heads=kv, mixers=mixers,
        layer_order=cfg.get("layer_order"),
    )
