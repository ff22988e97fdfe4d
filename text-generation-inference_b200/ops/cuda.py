"""ctypes bindings of the sm_100a kernel library (``libtgi_b200_kernels.so``, built by ``ops/build.py``).

Every wrapper allocates its outputs with torch (so they live in the caching allocator and are graph
capturable), passes raw pointers plus the current CUDA stream, and raises on a non-zero return code.
Kernels that wait on barriers report protocol time-outs through a device status word that
``check_status()`` reads; it is checked by tests and by the engine after each step, never inside a
captured graph.
"""
from __future__ import annotations

import ctypes
import os
from pathlib import Path
from typing import Optional, Tuple

import torch

_LIB = None
_LIB_PATH = Path(__file__).resolve().parent / "libtgi_b200_kernels.so"
FP8 = torch.float8_e4m3fn

_ACT_CODES = {"silu": 0, "swish": 0, "gelu": 1, "gelu_python": 1, "gelu_new": 2, "gelu_fast": 2,
              "gelu_pytorch_tanh": 2, "gelu_tanh": 2, "relu": 3, "quick_gelu": 4, "relu2": 5}

c_void_p, c_int, c_float, c_ll = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong


class KernelError(RuntimeError):
    pass


def lib_path() -> Path:
    return _LIB_PATH


def use_kernel_set(name: str) -> None:
    """Before the first kernel call: load the part ``name`` of the library (``build.KERNEL_SETS``), compiled now if need
    be, unless the whole library is there already."""
    global _LIB_PATH
    if _LIB is None and not _LIB_PATH.exists():
        from .build import build

        _LIB_PATH = build(kernel_set=name)


def load():
    """Load the kernel library; a missing library on a CUDA machine is an error, never a silent fallback."""
    global _LIB
    if _LIB is not None:
        return _LIB
    if not _LIB_PATH.exists():
        if os.environ.get("TGI_B200_AUTOBUILD", "1") == "1":
            from .build import build

            build()
        if not _LIB_PATH.exists():
            raise KernelError(
                f"{_LIB_PATH} is missing: build it with `python -m tgi_b200.ops.build` "
                "(the sm_100a kernels are required on CUDA devices)")
    _LIB = ctypes.CDLL(str(_LIB_PATH))
    for name in ("tgi_gemm_bf16", "tgi_gemm_fp8_block", "tgi_norm", "tgi_act_mul", "tgi_quant_act",
                 "tgi_rope_cache", "tgi_embedding", "tgi_argmax_logprob", "tgi_paged_attention", "tgi_paged_attention_ex",
                 "tgi_gemm_num_tiles", "tgi_attn_decode_splits", "tgi_attn_status", "tgi_lora_shrink",
                 "tgi_lora_expand", "tgi_moe_topk_softmax", "tgi_moe_sort", "tgi_moe_gather", "tgi_moe_grouped_gemm",
                 "tgi_moe_combine", "tgi_gemm_last_grid", "tgi_penalties", "tgi_gemm_wq", "tgi_wq_dequant", "tgi_qk_norm",
                 "tgi_quant_set_pow2", "tgi_peer_set_quant_pow2", "tgi_gemm_bf16_ld", "tgi_residual_norm", "tgi_embed_residual",
                 "tgi_activation", "tgi_attn_prep", "tgi_attn_any", "tgi_delta_prep", "tgi_delta_scan", "tgi_decay_scan",
                 "tgi_gated_norm", "tgi_recurrent_pitch", "tgi_delta_tap_rows", "tgi_act_mul_any", "tgi_moe_router",
                 "tgi_moe_router_splits", "tgi_moe_topk_sigmoid", "tgi_moe_topk_logits", "tgi_row_norm_store", "tgi_output_gate",
                 "tgi_map_store", "tgi_map_difference", "tgi_stream_step", "tgi_input_conv", "tgi_latent_store", "tgi_latent_rows", "tgi_latent_attention", "tgi_expanded_attention", "tgi_moe_grouped_f32", "tgi_moe_combine_f32"):
        if hasattr(_LIB, name):        # a library built for one family of models lacks the other families' kernels
            getattr(_LIB, name).restype = c_int
    _LIB.tgi_gemm_workspace_floats.restype = c_ll
    wide = os.environ.get("TGI_B200_GEMM_WIDE_M")
    if wide:
        _LIB.tgi_gemm_set_wide_m(c_int(int(wide)))
    if os.environ.get("TGI_B200_GEMM_PAIRS", "1") == "0":   # single-CTA 256 x 128 tiles instead of CTA pairs
        _LIB.tgi_gemm_set_pairs(c_int(0))
    if os.environ.get("TGI_B200_MX_PAIRS", "1") == "0":       # block-scaled mode on single CTAs only
        _LIB.tgi_gemm_set_mx_pairs(c_int(0))
    if os.environ.get("TGI_B200_GEMM_STREAMK_SMALL", "0") == "1":   # stream-K also below one tile per worker
        _LIB.tgi_gemm_set_streamk_small(c_int(1))
    # fp8 GEMMs run on the block-scaled MMA unless TGI_B200_FP8_MX=0 (then: per-K-block promotion, arbitrary scales)
    if os.environ.get("TGI_B200_FP8_MX", "1") == "1" and torch.cuda.is_available() and hasattr(_LIB, "tgi_peer_set_quant_pow2"):
        set_fp8_mx(True)
    return _LIB


_FP8_MX = False


def set_fp8_mx(on: bool) -> None:
    """Block-scaled fp8 GEMMs on ``tcgen05.mma.kind::mxf8f6f4``: the tensor core applies the block scales, so they
    must be powers of two.  Switching it on makes every activation-quantising kernel round its scales up to a power
    of two; block-scaled weights have to be brought to power-of-two scales once (``requant_block_pow2``, done by
    ``Fp8Linear`` at load)."""
    global _FP8_MX
    lib = _LIB if _LIB is not None else load()
    v = c_int(1 if on else 0)
    lib.tgi_gemm_set_fp8_mx(v)
    _check(lib.tgi_quant_set_pow2(v), "quant_set_pow2")
    _check(lib.tgi_peer_set_quant_pow2(v), "peer_set_quant_pow2")
    _FP8_MX = bool(on)
    from . import reference

    reference.POW2_ACT_SCALES = bool(on)     # the PyTorch oracle quantises the same way


def fp8_mx() -> bool:
    return _FP8_MX


def requant_block_pow2(wq: torch.Tensor, scale: torch.Tensor, block: int = 128):
    """e4m3 weights ``[N, K]`` with one scale per ``block x block`` tile -> the same matrix with every scale rounded
    up to a power of two and the values re-rounded to e4m3 (``w * s = w' * s'`` up to that rounding).  Engines that
    feed block-scaled checkpoints to Blackwell's scale-factor MMA do the same (it takes E8M0 scale factors)."""
    scale = scale.float()
    mant, expo = torch.frexp(scale)                      # scale = mant * 2^expo, mant in [0.5, 1)
    s2 = torch.where(mant == 0.5, scale, torch.ldexp(torch.ones_like(scale), expo))
    ratio = scale / s2                                   # in (0.5, 1]
    N, K = wq.shape
    out = torch.empty_like(wq)
    rows = max(block, (1 << 26) // max(K, 1) // block * block)     # chunks of about 64 M elements
    for r0 in range(0, N, rows):
        r1 = min(N, r0 + rows)
        rr = ratio[r0 // block:(r1 + block - 1) // block].repeat_interleave(block, 0)[:r1 - r0]
        rr = rr.repeat_interleave(block, 1)[:, :K]
        out[r0:r1] = (wq[r0:r1].float() * rr).to(wq.dtype)
    return out, s2.contiguous()


def set_gemm_pairs(on: bool) -> None:
    """Use CTA pairs (``cta_group::2``, 256 x 256 tiles) for GEMMs with more than 128 tokens (default), or
    single CTAs on 256 x 128 tiles."""
    load().tgi_gemm_set_pairs(c_int(1 if on else 0))


def _ptr(t: Optional[torch.Tensor]):
    return c_void_p(0 if t is None else t.data_ptr())


def _stream():
    return c_void_p(torch.cuda.current_stream().cuda_stream)


LAUNCHES = 0  # kernel-launching library calls made so far (benchmarks read and reset it)


def _check(rc: int, what: str):
    global LAUNCHES
    LAUNCHES += 1
    if rc != 0:
        raise KernelError(f"{what} failed with code {rc}")


# ---- per-device state: split-K workspace, counters, status word --------------------------------
class _DeviceState:
    def __init__(self, device: torch.device):
        self.device = device
        self.sm_count = torch.cuda.get_device_properties(device).multi_processor_count
        self.status = torch.zeros(1, dtype=torch.int32, device=device)
        self.counters = torch.zeros(1 << 16, dtype=torch.int32, device=device)
        self.ws = torch.empty(int(os.environ.get("TGI_B200_SPLITK_WS_MB", "64")) << 18, dtype=torch.float32,
                              device=device)
        self.attn_part_o = None
        self.attn_part_ml = None
        self.kept = {}


_STATES = {}


def state(device: torch.device) -> _DeviceState:
    idx = device.index if device.index is not None else torch.cuda.current_device()
    st = _STATES.get(idx)
    if st is None:
        st = _STATES[idx] = _DeviceState(torch.device("cuda", idx))
    return st


def check_status(device: Optional[torch.device] = None) -> int:
    """Read (and clear) the kernels' error word; 0 means no kernel gave up on a wait."""
    dev = device or torch.device("cuda", torch.cuda.current_device())
    st = state(dev)
    code = int(st.status.item())
    if code != 0:
        st.status.zero_()
        st.counters.zero_()    # a kernel that gave up may have left split-tile counters half-way
    with torch.cuda.device(st.device):
        attn = int(load().tgi_attn_status(c_int(1)))   # decode attention: a page copy did not arrive in time
    if attn != 0 and code == 0:
        code = 100 + attn
    return code


# ---- scale tensors -----------------------------------------------------------------------------
def alloc_act_scales(T: int, groups: int, device) -> torch.Tensor:
    """Activation scales, logical shape ``[T, groups]`` stored K-block major with a 16-byte aligned pitch."""
    pitch = (max(T, 1) + 3) & ~3
    buf = torch.empty(groups, pitch, dtype=torch.float32, device=device)
    return buf[:, :T].t()


def _scale_storage(xs: torch.Tensor) -> Tuple[int, int]:
    """(data_ptr, pitch) of a ``[T, groups]`` scale view produced by ``alloc_act_scales``."""
    if xs.dim() != 2 or (xs.shape[0] > 1 and xs.stride(0) != 1):
        raise KernelError("activation scales must be K-block major (use ops.fp8_quant_act / the fused producers)")
    pitch = xs.stride(1) if xs.shape[1] > 1 else ((xs.shape[0] + 3) & ~3)
    return xs.data_ptr(), pitch


# ---- GEMMs -------------------------------------------------------------------------------------
def _gemm_ctas(lib, st, M: int, N: int, max_ctas: Optional[int]) -> int:
    """Grid size of the persistent stream-K GEMM: one CTA per SM, bounded by the scratch buffers."""
    ctas = st.sm_count if max_ctas is None else max(1, min(int(max_ctas), st.sm_count))
    while ctas > 1 and lib.tgi_gemm_workspace_floats(M, ctas) > st.ws.numel():
        ctas -= 1
    if lib.tgi_gemm_num_tiles(M, N) > st.counters.numel():
        raise KernelError("GEMM has more output tiles than tile counters; raise the counter buffer size")
    return ctas


def gemm_bf16(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, max_ctas: Optional[int] = None,
              out: Optional[torch.Tensor] = None):
    lib = load()
    lead = x.shape[:-1]
    x2 = x if x.dim() == 2 else x.reshape(-1, x.shape[-1])
    # a column slice of a wider matrix is read in place when its rows start on 16-byte boundaries
    sliced = (x2.stride(1) == 1 and x2.stride(0) > x2.shape[1] and x2.stride(0) % 8 == 0 and x2.data_ptr() % 16 == 0
              and not getattr(out, "is_peer_push", False))
    if not sliced and not x2.is_contiguous():
        x2 = x2.contiguous()
    M, K = x2.shape
    N = w.shape[0]
    assert w.shape[1] == K and w.is_contiguous()
    if getattr(out, "is_peer_push", False):
        # row-parallel GEMM of a tensor-parallel group: rows go straight to their owners' peer memory
        if M == 0:
            return out
        assert out.T == M and out.N == N
        st = state(x.device)
        ctas = _gemm_ctas(lib, st, M, N, max_ctas)
        _check(lib.tgi_gemm_push(c_int(0), _ptr(x2), c_void_p(0), c_int(0), _ptr(w), c_void_p(0), _ptr(bias), c_int(M),
                                 c_int(N), c_int(K), c_int(ctas), _ptr(st.ws), _ptr(st.counters), _ptr(st.status),
                                 *out.gemm_args(), _stream()), "gemm_push")
        return out
    if out is None:
        out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    else:
        assert out.numel() == M * N and out.dtype == torch.bfloat16 and out.is_contiguous()
    if M == 0:
        return out.reshape(*lead, N)
    st = state(x.device)
    ctas = _gemm_ctas(lib, st, M, N, max_ctas)
    if sliced:
        _check(lib.tgi_gemm_bf16_ld(_ptr(x2), c_int(x2.stride(0)), _ptr(w), _ptr(out), _ptr(bias), c_int(M), c_int(N),
                                    c_int(K), c_int(ctas), _ptr(st.ws), _ptr(st.counters), _ptr(st.status), _stream()),
               "gemm_bf16_ld")
        return out.reshape(*lead, N)
    _check(lib.tgi_gemm_bf16(_ptr(x2), _ptr(w), _ptr(out), _ptr(bias), c_int(M), c_int(N), c_int(K), c_int(ctas),
                             _ptr(st.ws), _ptr(st.counters), _ptr(st.status), _stream()), "gemm_bf16")
    return out.reshape(*lead, N)


def gemm_fp8_block(xq, xs, wq, ws, out_dtype=torch.bfloat16, bias=None, max_ctas: Optional[int] = None, out=None):
    lib = load()
    M, K = xq.shape
    N = wq.shape[0]
    assert wq.shape[1] == K and wq.is_contiguous() and xq.is_contiguous()
    assert out_dtype == torch.bfloat16
    if getattr(out, "is_peer_push", False):
        if M == 0:
            return out
        assert out.T == M and out.N == N
        st = state(xq.device)
        sptr, pitch = _scale_storage(xs)
        ctas = _gemm_ctas(lib, st, M, N, max_ctas)
        if not ws.is_contiguous():
            ws = ws.contiguous()
        _check(lib.tgi_gemm_push(c_int(1), _ptr(xq), c_void_p(sptr), c_int(pitch), _ptr(wq), _ptr(ws), _ptr(bias),
                                 c_int(M), c_int(N), c_int(K), c_int(ctas), _ptr(st.ws), _ptr(st.counters),
                                 _ptr(st.status), *out.gemm_args(), _stream()), "gemm_push")
        return out
    if out is None:
        out = torch.empty(M, N, dtype=torch.bfloat16, device=xq.device)
    else:
        assert out.shape == (M, N) and out.dtype == torch.bfloat16 and out.is_contiguous()
    if M == 0:
        return out
    st = state(xq.device)
    sptr, pitch = _scale_storage(xs)
    ctas = _gemm_ctas(lib, st, M, N, max_ctas)
    if not ws.is_contiguous():
        ws = ws.contiguous()
    _check(lib.tgi_gemm_fp8_block(_ptr(xq), c_void_p(sptr), c_int(pitch), _ptr(wq), _ptr(ws), _ptr(out), _ptr(bias),
                                  c_int(M), c_int(N), c_int(K), c_int(ctas), _ptr(st.ws), _ptr(st.counters),
                                  _ptr(st.status), _stream()), "gemm_fp8_block")
    return out


# ---- norms -------------------------------------------------------------------------------------
def _norm(x, residual, weight, bias, eps, w_offset, layer, quant):
    lib = load()
    assert x.dtype == torch.bfloat16 and x.is_contiguous()
    T, H = x.shape
    res_out = torch.empty_like(x) if residual is not None else x
    out = q = scales = None
    if quant:
        q = torch.empty(T, H, dtype=FP8, device=x.device)
        scales = alloc_act_scales(T, H // 128, x.device)
        sptr, pitch = _scale_storage(scales)
    else:
        out = torch.empty_like(x)
        sptr, pitch = 0, 0
    _check(lib.tgi_norm(_ptr(x), _ptr(residual), _ptr(weight), _ptr(bias), _ptr(out),
                        _ptr(res_out if residual is not None else None), _ptr(q), c_void_p(sptr), c_int(pitch),
                        c_int(T), c_int(H), c_float(eps), c_float(w_offset), c_int(1 if layer else 0), _stream()),
           "norm")
    return out, q, scales, res_out


def rms_norm(x, residual, weight, eps, unit_offset=False):
    out, _, _, res = _norm(x, residual, weight, None, eps, 1.0 if unit_offset else 0.0, False, False)
    return out, res


def rms_norm_quant(x, residual, weight, eps, unit_offset=False):
    _, q, s, res = _norm(x, residual, weight, None, eps, 1.0 if unit_offset else 0.0, False, True)
    return q, s, res


def layer_norm(x, residual, weight, bias, eps):
    out, _, _, res = _norm(x, residual, weight, bias, eps, 0.0, True, False)
    return out, res


def qk_norm(qkv: torch.Tensor, num_heads: int, num_kv_heads: int, head_dim: int, q_weight: torch.Tensor,
            k_weight: torch.Tensor, eps: float, unit_offset: bool = False, layer: bool = False) -> torch.Tensor:
    """Per-head RMSNorm (or bias-free LayerNorm) of the q and k heads of ``qkv[T, (nh + 2 nkv) D]``, in place.  The
    weights are ``[D]`` (shared by the heads) or ``[heads, D]``."""
    lib = load()
    assert qkv.dtype == torch.bfloat16 and qkv.stride(1) == 1
    qw = q_weight.to(torch.bfloat16).contiguous()
    kw = k_weight.to(torch.bfloat16).contiguous()
    _check(lib.tgi_qk_norm(_ptr(qkv), c_ll(qkv.stride(0)), c_int(qkv.shape[0]), c_int(num_heads), c_int(num_kv_heads),
                           c_int(head_dim), _ptr(qw), _ptr(kw), c_int(head_dim if qw.dim() > 1 else 0),
                           c_int(head_dim if kw.dim() > 1 else 0), ctypes.c_float(eps),
                           ctypes.c_float(1.0 if unit_offset else 0.0), c_int(1 if layer else 0), _stream()), "qk_norm")
    return qkv


# ---- activation --------------------------------------------------------------------------------
def act_and_mul(gate_up, act="silu"):
    lib = load()
    T, I2 = gate_up.shape
    I = I2 // 2
    out = torch.empty(T, I, dtype=gate_up.dtype, device=gate_up.device)
    if gate_up.dtype == torch.float32 or I % 8 != 0:
        _check(lib.tgi_act_mul_any(_f32(gate_up), _ptr(gate_up.contiguous()), _ptr(out), c_int(T), c_int(I),
                                   c_int(_ACT_CODES[act]), _stream()), "act_and_mul")
        return out
    _check(lib.tgi_act_mul(_ptr(gate_up.contiguous()), _ptr(out), c_void_p(0), c_void_p(0), c_int(0), c_int(T),
                           c_int(I), c_int(_ACT_CODES[act]), _stream()), "act_and_mul")
    return out


def act_and_mul_quant(gate_up, act="silu"):
    lib = load()
    T, I2 = gate_up.shape
    I = I2 // 2
    q = torch.empty(T, I, dtype=FP8, device=gate_up.device)
    scales = alloc_act_scales(T, I // 128, gate_up.device)
    sptr, pitch = _scale_storage(scales)
    _check(lib.tgi_act_mul(_ptr(gate_up.contiguous()), c_void_p(0), _ptr(q), c_void_p(sptr), c_int(pitch), c_int(T),
                           c_int(I), c_int(_ACT_CODES[act]), _stream()), "act_and_mul_quant")
    return q, scales


def fp8_quant_act(x, group=128):
    lib = load()
    assert group == 128 and x.dtype == torch.bfloat16
    x = x.contiguous()
    T, K = x.shape
    q = torch.empty(T, K, dtype=FP8, device=x.device)
    scales = alloc_act_scales(T, K // 128, x.device)
    sptr, pitch = _scale_storage(scales)
    _check(lib.tgi_quant_act(_ptr(x), _ptr(q), c_void_p(sptr), c_int(pitch), c_int(T), c_int(K), _stream()),
           "fp8_quant_act")
    return q, scales


# ---- rope + cache ------------------------------------------------------------------------------
def rope_and_cache(qkv, positions, cos_sin, slots, k_cache, v_cache, num_heads, num_kv_heads, head_dim, rot_dim,
                   neox=True, k_scale=None, v_scale=None):
    lib = load()
    T = qkv.shape[0]
    qkv = qkv.contiguous()
    q = torch.empty(T, num_heads, head_dim, dtype=qkv.dtype, device=qkv.device)
    fp8 = k_cache.dtype == FP8
    num_slots = k_cache.shape[0] * k_cache.shape[1]
    _check(lib.tgi_rope_cache(_ptr(qkv), _ptr(positions), _ptr(cos_sin), _ptr(slots), _ptr(q), _ptr(k_cache),
                              _ptr(v_cache), _ptr(k_scale if fp8 else None), _ptr(v_scale if fp8 else None),
                              c_int(T), c_int(num_heads), c_int(num_kv_heads), c_int(head_dim), c_int(rot_dim),
                              c_int(1 if neox else 0), c_ll(num_slots), c_int(1 if fp8 else 0),
                              c_int(cos_sin.shape[0]), _stream()),
           "rope_and_cache")
    return q


# ---- attention ---------------------------------------------------------------------------------
ATTN_HEAD_DIMS = (64, 128, 256)      # head sizes of the tensor-core kernels (bf16 queries)


def attention_pitch(dim: int, vdim: int, dtype: torch.dtype) -> Tuple[int, int]:
    """Page widths ``(K, V)`` of a head with ``dim`` query/key and ``vdim`` value dimensions: both padded to one size of
    the tensor-core kernels where there is one, otherwise as they are (``tgi_attn_any``)."""
    if dtype == torch.bfloat16:
        for w in ATTN_HEAD_DIMS:
            if max(dim, vdim) <= w:
                return w, w
    return dim, vdim


def paged_attention(q, k_cache, v_cache, block_tables, cu_seqlens_q, kv_lens, scale, window=-1, softcap=0.0,
                    k_scale=None, v_scale=None, max_q=None, max_kv=None, nsplit: Optional[int] = None, horizon=None,
                    chunk: int = 0, sink=None, keep: int = 0):
    lib = load()
    if sink is False:
        sink = None
    elif sink is True:
        sink = _zero_sink(q.device, q.shape[1])
    assert sink is None or (sink.dtype == torch.float32 and sink.shape == (q.shape[1],) and sink.is_contiguous())
    T, Hq, D = q.shape
    nblk, bs, Hkv, _ = k_cache.shape
    Dv = v_cache.shape[3]
    B = kv_lens.shape[0]
    out = q.new_empty(T, Hq, Dv)
    if T == 0 or B == 0:
        return out
    if q.dtype == torch.float32 or D != Dv or D not in ATTN_HEAD_DIMS:
        assert horizon is None and k_cache.dtype == q.dtype and v_cache.dtype == q.dtype
        return _attention_any(q.contiguous(), k_cache, v_cache, Dv, block_tables, cu_seqlens_q, kv_lens, out, scale, softcap, window,
                              chunk, sink, None, keep)
    if max_q is None:
        max_q = int((cu_seqlens_q[1:] - cu_seqlens_q[:-1]).max().item())
    if max_kv is None:
        max_kv = int(kv_lens.max().item())
    for span in (chunk, window or 0):
        if span > 0:
            max_kv = min(max_kv, span + keep)   # keys a row can see: decides how far a decode step is split
    fp8 = k_cache.dtype == FP8
    st = state(q.device)
    part_o = part_ml = None
    if max_q == 1:
        if nsplit is None:
            nsplit = lib.tgi_attn_decode_splits(B, Hkv, Hq // Hkv, max_kv, st.sm_count)
        if nsplit > 1:
            need = B * Hq * nsplit
            part_o, part_ml = _attention_parts(st, need, D)
    else:
        nsplit = 1
    _check(lib.tgi_paged_attention_ex(
        _ptr(q.contiguous()), _ptr(k_cache), _ptr(v_cache), _ptr(block_tables), _ptr(cu_seqlens_q), _ptr(kv_lens),
        _ptr(k_scale if fp8 else None), _ptr(v_scale if fp8 else None), _ptr(out), _ptr(part_o), _ptr(part_ml),
        c_int(B), c_int(max_q), c_int(block_tables.shape[1]), c_int(bs), c_int(nblk), c_int(Hq), c_int(Hkv), c_int(D),
        c_float(scale), c_float(softcap), c_int(window if window and window > 0 else -1), c_int(chunk),
        c_int(keep), _ptr(sink), c_int(nsplit), c_int(1 if fp8 else 0), _ptr(horizon), _stream()), "paged_attention")
    return out


def _attention_parts(st, rows: int, D: int):
    """Workspace of a split decode step: partial outputs and their maxima and sums, each as large as it has to be (layers of
    other head sizes share them).  What captured steps use stays alive."""
    for name, need in (("attn_part_o", rows * D), ("attn_part_ml", rows * 2)):
        held = getattr(st, name)
        if held is None or held.numel() < need:
            if held is not None:
                st.kept.setdefault("outgrown", []).append(held)
            setattr(st, name, torch.empty(max(need, 2 * held.numel() if held is not None else 0), dtype=torch.float32, device=st.device))
    return st.attn_part_o, st.attn_part_ml


_ZERO_SINKS = {}


def _zero_sink(device, heads: int) -> torch.Tensor:
    """Scores of sinks that are 0 for every head (kept: captured decode steps read them)."""
    key = (device, heads)
    if key not in _ZERO_SINKS:
        _ZERO_SINKS[key] = torch.zeros(heads, dtype=torch.float32, device=device)
    return _ZERO_SINKS[key]


def _attention_any(q, k_cache, v_cache, vdim, block_tables, cu_seqlens_q, kv_lens, out, scale, softcap, window, chunk, sink, gate,
                   keep: int = 0):
    """The kernel for head sizes without an instance and for fp32; ``vdim`` columns of every value row are read."""
    T, Hq, D = q.shape
    _, bs, Hkv, ldv = v_cache.shape
    _check(load().tgi_attn_any(
        _f32(q), _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(block_tables), _ptr(cu_seqlens_q), _ptr(kv_lens), _ptr(out), c_int(T),
        c_int(kv_lens.shape[0]), c_int(block_tables.shape[1]), c_int(bs), c_int(Hq), c_int(Hkv), c_int(D), c_int(vdim), c_int(ldv),
        c_float(scale), c_float(softcap), c_int(window if window and window > 0 else -1), c_int(chunk), c_int(keep), _ptr(sink),
        _ptr(gate), c_ll(0 if gate is None else gate.stride(0)), _stream()), "attn_any")
    return out


def latent_layout(rank: int, rot: int, dtype: torch.dtype) -> Tuple[int, int]:
    """``(column of the rotated part, width)`` of a cached latent row: both parts start at multiples of 64 columns where the
    tensor-core kernel takes the row."""
    if dtype == torch.bfloat16:
        values, rotated = (rank + 63) // 64, (rot + 63) // 64
        if load().tgi_latent_rows(c_int(values + rotated), c_int(values), c_ll(1)) > 0:
            return 64 * values, 64 * (values + rotated)
    return rank, rank + rot


def expanded_dims(dim: int, vdim: int, dtype: torch.dtype):
    """``(query / key width, value width)`` of a head in ``expanded_attention``, ``None`` where it does not take the sizes."""
    if dtype != torch.bfloat16 or dim > 192 or vdim > 128:
        return None
    return (128 if dim <= 128 else 192), 128


def expanded_attention(q, kv, plan, cu_seqlens_q, scale, window, max_q: int, gate, out, sink=None):
    T, H, dk = q.shape
    R = kv.shape[0]
    assert q.is_contiguous() and out.is_contiguous() and tuple(out.shape) == (T, H, 128) and kv.is_contiguous()
    assert kv.shape[1] == H * (dk + 128) and R % 16 == 0 and (gate is None or gate.stride(1) == 1)
    st = state(q.device)
    _check(load().tgi_expanded_attention(
        _ptr(q), _ptr(kv), c_void_p(kv.data_ptr() + 2 * H * dk), c_ll(kv.stride(0)), _ptr(plan.tables), _ptr(cu_seqlens_q),
        _ptr(plan.kv_lens), _ptr(gate), c_ll(0 if gate is None else gate.stride(0)), _ptr(out), c_int(plan.kv_lens.shape[0]),
        c_int(max_q), c_int(plan.tables.shape[1]), c_int(R // 16), c_int(H), c_int(dk), c_float(scale),
        c_int(window if window and window > 0 else -1), _ptr(sink), _ptr(st.status), _stream()), "expanded_attention")


def latent_store(proj, off_c, weight, eps, positions, cos_sin, slots, pages, q, off_rot, rank: int, rot: int, heads: int, dim: int,
                 q_full=None, queries: bool = True, q_latent=None, width: Optional[int] = None):
    assert proj.stride(1) == 1 and cos_sin.shape[1] == rot
    assert pages is None or (pages.is_contiguous() and pages.shape[2] == 1 and pages.dtype == proj.dtype and weight.dtype == torch.float32)
    width = pages.shape[3] if pages is not None else width
    assert q is None or (q.is_contiguous() and q.shape[2] == width and q.dtype == proj.dtype)
    assert q_full is None or (q_full.is_contiguous() and q_full.dtype == proj.dtype)
    off_cq, cq_weight, cq = q_latent or (0, None, None)
    assert cq is None or (cq.is_contiguous() and cq.dtype == proj.dtype and cq_weight.dtype == torch.float32)
    _check(load().tgi_latent_store(
        _f32(proj), _ptr(proj), c_ll(proj.stride(0)), c_int(off_c), _ptr(weight), c_float(eps), _ptr(positions), _ptr(cos_sin),
        c_int(cos_sin.shape[0]), _ptr(slots), _ptr(pages), c_ll(0 if pages is None else pages.shape[0] * pages.shape[1]),
        _ptr(proj if queries else None), c_ll(proj.stride(0)), _ptr(q), _ptr(q_full), c_int(off_cq),
        c_int(0 if cq is None else cq_weight.shape[0]), _ptr(cq_weight), _ptr(cq), c_int(0 if cq is None else cq.shape[1]),
        c_int(proj.shape[0]), c_int(heads), c_int(dim), c_int(rank), c_int(rot), c_int(off_rot), c_int(width),
        c_int(0 if q_full is None else q_full.shape[2]), _stream()), "latent_store")


def latent_attention(q, pages, rank: int, block_tables, cu_seqlens_q, kv_lens, scale, window=-1, max_q=None, max_kv=None, gate=None,
                     elsewhere=None, sink=None):
    """Tensor-core kernel for bf16 rows in 64-column pieces on pages of 16 tokens, ``tgi_attn_any`` otherwise."""
    lib = load()
    T, H, width = q.shape
    B = kv_lens.shape[0]
    assert gate is None or (gate.stride(1) == 1 and gate.dtype == q.dtype)
    assert sink is None or (sink.dtype == torch.float32 and sink.shape == (H,) and sink.is_contiguous())
    assert q.is_contiguous() and pages.is_contiguous() and pages.shape[3] == width and pages.dtype == q.dtype
    values = (rank + 63) // 64
    if q.dtype == torch.bfloat16 and width % 64 == 0 and pages.shape[1] == 16 and max_q is not None:
        N = int(lib.tgi_latent_rows(c_int(width // 64), c_int(values), c_ll(max_q * H)))
        if N > 0:
            out = q.new_empty(T, H, 64 * values)
            st = state(q.device)
            part = _latent_parts(st, N, 64 * values, B * ((H + N - 1) // N)) if max_q == 1 else (None,) * 3
            _check(lib.tgi_latent_attention(
                _ptr(q), _ptr(pages), _ptr(block_tables), _ptr(cu_seqlens_q), _ptr(kv_lens), _ptr(gate),
                c_ll(0 if gate is None else gate.stride(0)), _ptr(sink), _ptr(out), *map(_ptr, part), c_int(T), c_int(B), c_int(max_q),
                c_int(block_tables.shape[1]), c_int(pages.shape[0]), c_int(H), c_int(width // 64), c_int(values), c_int(N),
                c_float(scale), c_int(window if window and window > 0 else -1), _ptr(elsewhere), c_int(st.sm_count),
                _ptr(st.status), _stream()), "latent_attention")
            return out
    assert elsewhere is None
    out = q.new_empty(T, H, rank)
    if T == 0:
        return out
    return _attention_any(q, pages, pages, rank, block_tables, cu_seqlens_q, kv_lens, out, scale, 0.0, window, 0, sink, gate)


def _latent_parts(st, N: int, cols: int, items: int):
    """Workspace of a persistent latent attention (kept: captured decode steps use it)."""
    key = ("latent", N, cols)
    if key not in st.kept:
        st.kept[key] = (torch.empty(2 * st.sm_count * N * cols, dtype=torch.float32, device=st.device),
                        torch.empty(2 * st.sm_count * N * 2, dtype=torch.float32, device=st.device))
    items = max(1024, 1 << (items - 1).bit_length())
    if ("range", items) not in st.kept:
        st.kept["range", items] = torch.zeros(2 * items, dtype=torch.int32, device=st.device)
    return (*st.kept[key], st.kept["range", items])


def row_norm_store(proj, offs, positions, slots, k_cache, v_cache, q_weight, k_weight, eps, num_heads: int, num_kv_heads: int,
                   dim: int, vdim: int, width: int, temperature=None):
    T = proj.shape[0]
    q = torch.empty(T, num_heads, width, dtype=proj.dtype, device=proj.device)
    assert proj.stride(1) == 1 and k_cache.dtype == proj.dtype and v_cache.dtype == proj.dtype
    coef, every = temperature or (0.0, 0)
    off_k, off_v = (offs[1], offs[2]) if k_weight is not None else (0, 0)
    _check(load().tgi_row_norm_store(
        _f32(proj), _ptr(proj), c_ll(proj.stride(0)), c_int(off_k), c_int(off_v), _ptr(positions), _ptr(slots), _ptr(q_weight),
        _ptr(k_weight), _ptr(q), _ptr(k_cache), _ptr(v_cache), c_int(T), c_int(num_heads), c_int(num_kv_heads), c_int(dim),
        c_int(vdim), c_int(width), c_int(k_cache.shape[3]), c_int(v_cache.shape[3]), c_ll(k_cache.shape[0] * k_cache.shape[1]),
        c_float(eps), c_float(coef), c_int(every), _stream()), "row_norm_store")
    return q


def map_store(proj, offs, slots, k_cache, v_cache, num_heads: int, num_kv_heads: int, dim: int, vdim: int):
    T, Dk, Dv = proj.shape[0], k_cache.shape[3], v_cache.shape[3]
    q = torch.empty(T, 2 * num_heads, Dk, dtype=proj.dtype, device=proj.device)
    assert proj.stride(1) == 1 and k_cache.dtype == proj.dtype and v_cache.dtype == proj.dtype and offs[0] == 0
    assert k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.shape[2] == v_cache.shape[2] == num_kv_heads
    _check(load().tgi_map_store(
        _f32(proj), _ptr(proj), c_ll(proj.stride(0)), c_int(offs[1]), c_int(offs[2]), _ptr(slots), _ptr(q), _ptr(k_cache),
        _ptr(v_cache), c_int(T), c_int(num_heads), c_int(num_kv_heads), c_int(dim), c_int(vdim), c_int(Dk), c_int(Dv),
        c_ll(k_cache.shape[0] * k_cache.shape[1]), _stream()), "map_store")
    return q


def map_difference(a, gate, lam: float, factor: float, eps: float, width: int):
    T, H2, pitch = a.shape
    out = torch.empty(T, H2 // 2 * width, dtype=a.dtype, device=a.device)
    assert a.is_contiguous() and H2 % 2 == 0 and (gate is None or (gate.stride(1) == 1 and gate.dtype == a.dtype))
    _check(load().tgi_map_difference(
        _f32(a), _ptr(a), _ptr(gate), c_ll(0 if gate is None else gate.stride(0)), _ptr(out), c_int(T), c_int(H2 // 2), c_int(pitch),
        c_int(width), c_float(lam), c_float(factor), c_float(eps), _stream()), "map_difference")
    return out


def output_gate(x, gate, width: int):
    T, H, pitch = x.shape
    out = torch.empty(T, H * width, dtype=x.dtype, device=x.device)
    assert x.is_contiguous() and gate.stride(1) == 1 and gate.dtype == x.dtype
    _check(load().tgi_output_gate(_f32(x), _ptr(x), _ptr(gate), c_ll(gate.stride(0)), _ptr(out), c_int(T), c_int(H), c_int(pitch),
                                  c_int(width), _stream()), "output_gate")
    return out


# ---- token mixers of hybrid decoders -------------------------------------------------------------
def _f32(t: torch.Tensor):
    if t.dtype not in (torch.float32, torch.bfloat16):
        raise KernelError(f"hybrid decoders run in bfloat16 or float32, not {t.dtype}")
    return c_int(1 if t.dtype == torch.float32 else 0)


def embed_residual(ids, table, scale: float, streams: int = 1):
    T, H = ids.numel(), table.shape[1]
    out = torch.empty(*((streams, T, H) if streams > 1 else (T, H)), dtype=torch.float32, device=table.device)
    _check(load().tgi_embed_residual(_f32(table), _ptr(ids), _ptr(table), _ptr(out), c_int(T), c_int(H),
                                     c_int(table.shape[0]), c_float(scale), _stream()), "embed_residual")
    return out


def residual_norm(delta, residual, weight, eps, rows=None, keep: bool = True, scale: float = 1.0, unit_offset: bool = False,
                  weight2=None, layer: bool = False, bias=None):
    H = residual.shape[1]
    n = residual.shape[0] if rows is None else rows.shape[0]
    d1, d2 = delta if isinstance(delta, tuple) else (delta, None)
    new = lambda: torch.empty(n, H, dtype=weight.dtype, device=residual.device)
    out, out2 = new(), new() if weight2 is not None else None
    if d1 is None and rows is None:
        res = None if not keep else residual
        dst = None
    else:
        res = dst = torch.empty(n, H, dtype=torch.float32, device=residual.device) if keep else None
    assert residual.dtype == torch.float32 and residual.is_contiguous()
    assert bias is None or bias.dtype == weight.dtype
    assert all(d is None or (d.dtype == weight.dtype and d.is_contiguous() and d.shape == residual.shape) for d in (d1, d2))
    _check(load().tgi_residual_norm(_f32(weight), _ptr(d1), _ptr(d2), _ptr(residual), _ptr(rows), _ptr(weight), _ptr(weight2),
                                    _ptr(bias), _ptr(out), _ptr(out2), _ptr(dst), c_int(n), c_int(H), c_int(1 if layer else 0),
                                    c_float(eps), c_float(scale),
                                    c_float(1.0 if unit_offset else 0.0), _stream()), "residual_norm")
    return (out, res) if weight2 is None else (out, out2, res)


def _conv_args(conv, H: int, dtype):
    if conv is None:
        return [_ptr(None)] * 5 + [c_int(0)] * 3
    taps = conv.state.shape[1] + 1
    assert conv.weights.is_contiguous() and conv.weights.dtype == torch.float32 and tuple(conv.weights.shape) == (taps, H)
    assert conv.state.is_contiguous() and conv.state.shape[2] == H and conv.state.dtype == dtype
    return [*map(_ptr, (conv.weights, conv.cu, conv.kv_lens, conv.state_slots, conv.state)), c_int(conv.kv_lens.shape[0]),
            c_int(taps), c_int(conv.state.shape[0])]


def stream_step(delta, post, residual, weight, eps, rows=None, keep: bool = True, gain: float = 1.0, average=None, streams=None,
                conv=None):
    T, H = residual.shape
    n = T if rows is None else rows.shape[0]
    out = torch.empty(n, H, dtype=weight.dtype, device=residual.device)
    changed = delta is not None or average is not None or rows is not None
    res = dst = torch.empty(n, H, dtype=torch.float32, device=residual.device) if keep and changed else None
    if keep and not changed:
        res = residual
    assert residual.dtype == torch.float32 and residual.is_contiguous()
    assert delta is None or (delta.dtype == weight.dtype and delta.is_contiguous() and delta.shape == residual.shape)
    assert post is None or (post.dtype == weight.dtype and post.shape == (H,))
    index = 0
    if average is None:
        streams = None
    else:
        index = average.shape[0] - 1
        assert average.dtype == torch.float32 and streams.dtype == torch.float32 and streams.is_contiguous()
        assert streams.shape[1:] == residual.shape and index < streams.shape[0]
    _check(load().tgi_stream_step(
        _f32(weight), _ptr(delta), _ptr(post), _ptr(residual), _ptr(rows), _ptr(streams), _ptr(average), c_ll(T * H), c_int(index),
        c_int(1 if rows is None else 0), _ptr(weight), c_float(gain), _ptr(out), _ptr(dst), c_int(n), c_int(H), c_float(eps),
        *_conv_args(conv, H, weight.dtype), _stream()), "stream_step")
    return out, res


def input_conv(x, conv):
    out = torch.empty_like(x)
    assert x.is_contiguous()
    _check(load().tgi_input_conv(_f32(x), _ptr(x), _ptr(out), c_int(x.shape[0]), c_int(x.shape[1]), *_conv_args(conv, x.shape[1], x.dtype),
                                 _stream()), "input_conv")
    return out


def activation(x, act: str):
    out = torch.empty_like(x)
    _check(load().tgi_activation(_f32(x), _ptr(x), _ptr(out), c_ll(x.numel()), c_int(_ACT_CODES[act]), _stream()),
           "activation")
    return out


def rotate_norm_store(proj, offs, positions, cos_sin, slots, k_cache, v_cache, num_heads, num_kv_heads, dim, vdim, rot_dim,
                      qk_norm, eps, v_first=None, v_lambda: float = 0.0, interleaved: bool = False, conv=None):
    T = proj.shape[0]
    Dk, Dv = k_cache.shape[3], v_cache.shape[3]
    q = torch.empty(T, num_heads, Dk, dtype=proj.dtype, device=proj.device)
    assert proj.stride(1) == 1 and k_cache.dtype == proj.dtype and v_cache.dtype == proj.dtype
    assert v_first is None or (v_first.stride(1) == 1 and v_first.shape[1] == num_kv_heads * vdim and v_first.dtype == proj.dtype)
    past = [None] * 5 + [0] * 4
    if conv is not None:
        taps, channels = conv.state.shape[1] + 1, (num_heads + num_kv_heads) * dim + num_kv_heads * vdim
        assert conv.weights.is_contiguous() and tuple(conv.weights.shape) == (conv_rows(taps), channels)
        assert conv.state.is_contiguous() and conv.state.shape[2] == channels and conv.state.dtype == proj.dtype
        past = [conv.weights, conv.cu, conv.kv_lens, conv.state_slots, conv.state, conv.kv_lens.shape[0], taps,
                conv.state.shape[0], int(conv.single)]
    _check(load().tgi_attn_prep(
        _f32(proj), _ptr(proj), c_ll(proj.stride(0)), c_int(offs[1]), c_int(offs[2]), _ptr(positions), _ptr(cos_sin),
        _ptr(slots), _ptr(v_first), c_ll(0 if v_first is None else v_first.stride(0)), c_float(v_lambda), _ptr(q),
        _ptr(k_cache), _ptr(v_cache), c_int(T), c_int(num_heads), c_int(num_kv_heads), c_int(dim), c_int(vdim),
        c_int(Dk), c_int(Dv), c_int(rot_dim), c_int(cos_sin.shape[0]), c_ll(k_cache.shape[0] * k_cache.shape[1]),
        c_int(1 if qk_norm else 0), c_float(eps), c_int(1 if interleaved else 0), *map(_ptr, past[:5]),
        *map(c_int, past[5:]), _stream()), "attn_prep")
    return q


def recurrent_pitch(dim: int) -> int:
    w = int(load().tgi_recurrent_pitch(c_int(dim)))
    if w == 0:
        raise KernelError(f"recurrent heads of {dim} key channels are wider than the kernels support (256)")
    return w


def conv_rows(taps: int) -> int:
    return int(load().tgi_delta_tap_rows(c_int(taps)))


def delta_inputs(proj, offs, a_pre, conv_t, a_log, dt_bias, cu, kv_lens, state_slots, conv_state, kv_heads, heads, dim,
                 pitch, vdim, single: bool, head_decay: bool = False):
    T, dev = proj.shape[0], proj.device
    new = lambda *shape: torch.empty(*shape, dtype=torch.float32, device=dev)
    q, k = new(T, kv_heads, pitch), new(T, kv_heads, pitch)
    g = new(T, heads) if head_decay else new(T, heads, pitch)
    v, beta, qk = new(T, heads, vdim), new(T, heads), new(T, kv_heads)
    taps = conv_state.shape[1] + 1
    assert proj.stride(1) == 1 and a_pre.stride(1) == 1 and conv_state.dtype == proj.dtype
    assert conv_t.is_contiguous() and tuple(conv_t.shape) == (conv_rows(taps), conv_state.shape[2])
    _check(load().tgi_delta_prep(
        _f32(proj), _ptr(proj), c_ll(proj.stride(0)), c_int(offs[0]), c_int(offs[1]), c_int(offs[2]), c_int(offs[3]),
        _ptr(a_pre), c_ll(a_pre.stride(0)), _ptr(conv_t), _ptr(a_log), _ptr(dt_bias), _ptr(cu),
        _ptr(kv_lens), _ptr(state_slots), _ptr(conv_state), _ptr(q), _ptr(k), _ptr(v), _ptr(g), _ptr(beta), _ptr(qk),
        c_int(T), c_int(kv_lens.shape[0]), c_int(conv_state.shape[0]), c_int(kv_heads), c_int(heads), c_int(dim),
        c_int(pitch), c_int(vdim), c_int(taps), c_int(1 if single else 0), c_int(1 if head_decay else 0), _stream()),
        "delta_prep")
    return q, k, v, g, beta, qk


def delta_scan(q, k, v, g, beta, qk, cu, kv_lens, state_slots, state, dim: int, max_q: int):
    T, heads, vdim = v.shape
    out = torch.empty(T, heads, vdim, dtype=torch.float32, device=v.device)
    _check(load().tgi_delta_scan(
        _ptr(q), _ptr(k), _ptr(g), _ptr(v), _ptr(beta), _ptr(qk), _ptr(cu), _ptr(kv_lens), _ptr(state_slots), _ptr(state),
        _ptr(out), c_int(kv_lens.shape[0]), c_int(max_q), c_int(state.shape[0]), c_int(k.shape[1]), c_int(heads), c_int(dim),
        c_int(state.shape[3]), c_int(vdim), c_int(1 if g.dim() == 2 else 0), _stream()), "delta_scan")
    return out


def decay_scan(proj, offs, decay, cu, kv_lens, state_slots, state, heads: int, dim: int, vdim: int, max_q: int,
               act: str = "silu", k_scale: float = 1.0):
    T = proj.shape[0]
    out = torch.empty(T, heads, vdim, dtype=torch.float32, device=proj.device)
    _check(load().tgi_decay_scan(
        _f32(proj), _ptr(proj), c_ll(proj.stride(0)), c_int(offs[0]), c_int(offs[1]), c_int(offs[2]), _ptr(decay), _ptr(cu),
        _ptr(kv_lens), _ptr(state_slots), _ptr(state), _ptr(out), c_int(kv_lens.shape[0]), c_int(max_q),
        c_int(state.shape[0]), c_int(heads), c_int(dim), c_int(state.shape[3]), c_int(vdim), c_int({"silu": 1, "": 0}[act]),
        c_float(k_scale), _stream()), "decay_scan")
    return out


def gated_norm(o, gate, weight, eps, groups: int, out_cols: int, act: str = "sigmoid"):
    T = o.shape[0]
    width = o.numel() // max(T * groups, 1)
    out = torch.empty(T, out_cols, dtype=gate.dtype, device=o.device)
    assert gate.stride(1) == 1 and weight.dtype == torch.float32
    _check(load().tgi_gated_norm(_f32(gate), _ptr(o), _ptr(gate), c_ll(gate.stride(0)), c_int(0), _ptr(weight), _ptr(out),
                                 c_ll(out_cols), c_int(T), c_int(groups), c_int(width), c_float(eps),
                                 c_int({"sigmoid": 0, "silu": 1}[act]), _stream()), "gated_norm")
    return out


# ---- misc --------------------------------------------------------------------------------------
def embedding(ids, table):
    lib = load()
    if table.dtype != torch.bfloat16:
        return torch.nn.functional.embedding(ids.long(), table)
    T = ids.numel()
    ids32 = ids if ids.dtype == torch.int32 else ids.to(torch.int32)
    out = torch.empty(T, table.shape[1], dtype=table.dtype, device=table.device)
    _check(lib.tgi_embedding(_ptr(ids32.contiguous()), _ptr(table), _ptr(out), c_int(T), c_int(table.shape[1]),
                             c_int(table.shape[0]), _stream()), "embedding")
    return out.view(*ids.shape, table.shape[1])


def argmax_logprob(logits):
    lib = load()
    assert logits.dim() == 2 and logits.stride(1) == 1
    B, V = logits.shape
    if logits.dtype not in (torch.bfloat16, torch.float32):
        logits = logits.float()
    ids = torch.empty(B, dtype=torch.int64, device=logits.device)
    lp = torch.empty(B, dtype=torch.float32, device=logits.device)
    _check(lib.tgi_argmax_logprob(_ptr(logits), _ptr(ids), _ptr(lp), c_int(B), c_int(V), c_ll(logits.stride(0)),
                                  c_int(1 if logits.dtype == torch.float32 else 0), _stream()), "argmax_logprob")
    return ids, lp


def fused_sample(scores: torch.Tensor, temperature=None, top_k=None, top_p=None, do_sample=None, seeds=None, steps=None,
                 typical_p=None):
    """Temperature, top-k, top-p and sampling (Gumbel-max with a counter-based generator keyed by the
    request's seed and step) in one kernel; returns ``(ids int64 [B], logprobs fp32 [B])``.  Any stage
    whose tensor is ``None`` is off; rows with ``do_sample == 0`` take the argmax of the filtered scores."""
    lib = load()
    assert scores.dim() == 2 and scores.stride(1) == 1 and scores.dtype in (torch.float32, torch.bfloat16)
    B, V = scores.shape
    dev = scores.device
    ids = torch.empty(B, dtype=torch.int64, device=dev)
    lps = torch.empty(B, dtype=torch.float32, device=dev)
    if B == 0:
        return ids, lps

    def as_(t, dtype):
        return None if t is None else t.to(device=dev, dtype=dtype).contiguous()

    temperature, top_p = as_(temperature, torch.float32), as_(top_p, torch.float32)
    typical_p = as_(typical_p, torch.float32)
    top_k, steps = as_(top_k, torch.int32), as_(steps, torch.int32)
    do_sample, seeds = as_(do_sample, torch.uint8), as_(seeds, torch.int64)
    _check(lib.tgi_sample(_ptr(scores), c_ll(scores.stride(0)), c_int(1 if scores.dtype == torch.float32 else 0),
                          _ptr(temperature), _ptr(top_k), _ptr(top_p), _ptr(typical_p), _ptr(do_sample), _ptr(seeds),
                          _ptr(steps), _ptr(ids), _ptr(lps), c_int(B), c_int(V), _stream()), "sample")
    return ids, lps


# ---- weight-only quantised GEMM ------------------------------------------------------------------
_WQ_SCRATCH = {}


def _wq_partial(device) -> torch.Tensor:
    """fp32 workspace of the K-split partial tiles (shared by all layers of a device)."""
    key = ("partial", device.index)
    t = _WQ_SCRATCH.get(key)
    if t is None:
        t = torch.empty(int(os.environ.get("TGI_B200_WQ_WS_MB", "64")) << 18, dtype=torch.float32, device=device)
        _WQ_SCRATCH[key] = t
    return t


def gemm_wq(x: torch.Tensor, wq: torch.Tensor, scale: torch.Tensor, zp: Optional[torch.Tensor], group: int, bits: int,
            bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``x[M, K] (bf16) @ dequant(wq)[N, K]^T`` with the weights dequantised on their way into shared memory:
    ``wq`` uint8 ``[N, K/2]`` (4-bit, low nibble first) or int8 ``[N, K]``; ``scale`` / ``zp`` fp16 ``[K/group, N]``."""
    lib = load()
    st = state(x.device)
    M, K = x.shape
    N = wq.shape[0]
    out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    part = _wq_partial(x.device)
    x = x.contiguous()
    xh = torch.empty(M, K, dtype=torch.float16, device=x.device)       # fp16 copy of the tokens, written by the call
    _check(lib.tgi_gemm_wq(c_int(bits), _ptr(x), _ptr(xh), _ptr(wq), _ptr(scale), _ptr(zp), c_int(group), _ptr(out),
                           _ptr(part), c_ll(part.numel()), _ptr(bias), c_int(M), c_int(N), c_int(K), c_int(st.sm_count),
                           _ptr(st.status), _stream()), "gemm_wq")
    return out


def wq_dequant(wq: torch.Tensor, scale: torch.Tensor, zp: Optional[torch.Tensor], group: int, bits: int, K: int,
               out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """bf16 ``[N, K]`` matrix of a packed weight (the numbers the fused GEMM feeds to the tensor cores)."""
    lib = load()
    N = wq.shape[0]
    if out is None:
        out = torch.empty(N, K, dtype=torch.bfloat16, device=wq.device)
    _check(lib.tgi_wq_dequant(c_int(bits), _ptr(wq), _ptr(scale), _ptr(zp), c_int(group), _ptr(out), c_int(N), c_int(K),
                              _stream()), "wq_dequant")
    return out


def wq_dequant_scratch(wq, scale, zp, group, bits, K) -> torch.Tensor:
    """Dequantise into a per-device scratch matrix that the next call overwrites (prefill-sized GEMMs)."""
    N = wq.shape[0]
    key = ("dequant", wq.device.index)
    t = _WQ_SCRATCH.get(key)
    if t is None or t.numel() < N * K:
        t = torch.empty(N * K, dtype=torch.bfloat16, device=wq.device)
        _WQ_SCRATCH[key] = t
    return wq_dequant(wq, scale, zp, group, bits, K, out=t[: N * K].view(N, K))


def penalties(logits: torch.Tensor, history: torch.Tensor, repetition_penalty: Optional[torch.Tensor],
              frequency_penalty: Optional[torch.Tensor], vocab_start: int = 0, logit_scale: float = 1.0) -> torch.Tensor:
    """fp32 copy of ``logits[B, V]`` (bf16 or fp32; ``V`` may be a vocabulary slice starting at ``vocab_start``) with
    the repetition and frequency penalties of the rows' token ``history[B, L]`` applied, in one kernel."""
    lib = load()
    B, V = logits.shape
    assert logits.stride(1) == 1 and logits.dtype in (torch.bfloat16, torch.float32)
    out = torch.empty(B, V, dtype=torch.float32, device=logits.device)
    history = history.to(device=logits.device, dtype=torch.int64).contiguous()
    rep = None if repetition_penalty is None else repetition_penalty.to(torch.float32).contiguous()
    freq = None if frequency_penalty is None else frequency_penalty.to(torch.float32).contiguous()
    _check(lib.tgi_penalties(_ptr(logits), c_int(1 if logits.dtype == torch.float32 else 0), c_ll(logits.stride(0)),
                             _ptr(out), c_ll(V), _ptr(history), c_int(history.shape[1]), _ptr(rep), _ptr(freq),
                             c_int(vocab_start), c_int(B), c_int(V), ctypes.c_float(logit_scale), _stream()), "penalties")
    return out


def moe_topk_softmax(router_logits: torch.Tensor, top_k: int, renormalize: bool = True):
    """Softmax over the router logits and top-k selection in one kernel: ``(weights fp32 [T, k], ids int32 [T, k])``."""
    lib = load()
    T, E = router_logits.shape
    if router_logits.dtype not in (torch.float32, torch.bfloat16):
        router_logits = router_logits.float()
    router_logits = router_logits.contiguous()
    w = torch.empty(T, top_k, dtype=torch.float32, device=router_logits.device)
    ids = torch.empty(T, top_k, dtype=torch.int32, device=router_logits.device)
    _check(lib.tgi_moe_topk_softmax(_ptr(router_logits), c_int(1 if router_logits.dtype == torch.float32 else 0), c_int(T),
                                    c_int(E), c_int(top_k), c_int(1 if renormalize else 0), _ptr(w), _ptr(ids), _stream()),
           "moe_topk_softmax")
    return w, ids


def moe_experts(x, w_gate_up, w_down, topk_weights, topk_ids, act="silu", first: int = 0):
    """Routed expert MLPs of the experts ``first .. first + E_local - 1`` held in ``w_gate_up [E_local, 2I, H]`` /
    ``w_down [E_local, H, I]``: ``out[t] = sum_slot w[t, slot] * MLP_{id[t, slot]}(x[t])`` over the slots whose
    expert is local.  Five launches (group, gather, two grouped tcgen05 GEMMs with the activation and the routing
    weight fused into their epilogues, combine), no host synchronisation, fixed buffer shapes: the whole sequence
    is CUDA-graph capturable and only routed rows are computed."""
    lib = load()
    st = state(x.device)
    T, H = x.shape
    E_local, I2, _ = w_gate_up.shape
    I = I2 // 2
    k = topk_ids.shape[1]
    entries = T * k
    dev = x.device
    if T == 0:
        return torch.zeros(0, H, dtype=x.dtype, device=dev)
    assert x.dtype == torch.bfloat16 and w_gate_up.dtype == torch.bfloat16 and w_down.dtype == torch.bfloat16
    assert w_gate_up.is_contiguous() and w_down.is_contiguous() and tuple(w_down.shape) == (E_local, H, I)
    ids = topk_ids.to(torch.int32).contiguous()
    tw = topk_weights.to(torch.float32).contiguous()
    pos = torch.empty(entries, dtype=torch.int32, device=dev)
    order = torch.empty(entries, dtype=torch.int32, device=dev)
    offsets = torch.empty(E_local + 1, dtype=torch.int32, device=dev)
    grouped = torch.empty(entries, H, dtype=torch.bfloat16, device=dev)
    hidden = torch.empty(entries, I, dtype=torch.bfloat16, device=dev)
    y = torch.empty(entries, H, dtype=torch.bfloat16, device=dev)
    out = torch.empty(T, H, dtype=torch.bfloat16, device=dev)
    s = _stream()
    x = x.contiguous()
    _check(lib.tgi_moe_sort(_ptr(ids), c_int(entries), c_int(first), c_int(E_local), _ptr(pos), _ptr(order), _ptr(offsets),
                            s), "moe_sort")
    _check(lib.tgi_moe_gather(_ptr(x), _ptr(order), _ptr(offsets), c_int(E_local), c_int(k), c_int(H), c_int(entries),
                              _ptr(grouped), s), "moe_gather")
    _check(lib.tgi_moe_grouped_gemm(c_int(0), _ptr(grouped), c_int(entries), _ptr(w_gate_up), c_int(E_local), c_int(I2),
                                    c_int(H), _ptr(offsets), c_int(_ACT_CODES[act]), c_void_p(0), c_void_p(0),
                                    _ptr(hidden), c_int(st.sm_count), _ptr(st.status), s), "moe_grouped_gemm(gate_up)")
    _check(lib.tgi_moe_grouped_gemm(c_int(1), _ptr(hidden), c_int(entries), _ptr(w_down), c_int(E_local), c_int(H),
                                    c_int(I), _ptr(offsets), c_int(0), _ptr(tw), _ptr(order), _ptr(y),
                                    c_int(st.sm_count), _ptr(st.status), s), "moe_grouped_gemm(down)")
    _check(lib.tgi_moe_combine(_ptr(y), _ptr(pos), c_int(T), c_int(k), c_int(H), _ptr(out), s), "moe_combine")
    return out


def _router_logits(x, weight):
    """``x @ weight^T`` in fp32 as partial sums ``[parts, T, E]`` over ranges of K, and their number."""
    lib = load()
    T, E = x.shape[0], weight.shape[0]
    if x.dtype == torch.bfloat16:
        K = weight.shape[1]                    # rows of 16-byte pieces: padded at load where the width is no multiple of 8
        x = torch.nn.functional.pad(x, (0, K - x.shape[1])) if K > x.shape[1] else x.contiguous()
        splits = int(lib.tgi_moe_router_splits(c_int(T), c_int(E), c_int(K), c_int(state(x.device).sm_count)))
        part = torch.empty(splits, T, E, dtype=torch.float32, device=x.device)
        assert weight.is_contiguous() and weight.dtype == x.dtype
        _check(lib.tgi_moe_router(_ptr(x), _ptr(weight), c_int(T), c_int(E), c_int(K), c_int(splits), _ptr(part), _stream()),
               "moe_router")
    else:
        part, splits = torch.nn.functional.linear(x, weight), 1
    return part, splits


def moe_route_sigmoid(x, weight, correction, top_k: int, scale: float):
    """Router logits ``x @ weight^T`` in fp32, experts chosen by ``sigmoid + correction``, weights ``scale * s / sum(s)``."""
    T, E = x.shape[0], weight.shape[0]
    part, splits = _router_logits(x, weight)
    w = torch.empty(T, top_k, dtype=torch.float32, device=x.device)
    ids = torch.empty(T, top_k, dtype=torch.int32, device=x.device)
    _check(load().tgi_moe_topk_sigmoid(_ptr(part), c_int(splits), _ptr(correction), c_int(T), c_int(E), c_int(top_k), c_float(scale),
                                       _ptr(w), _ptr(ids), _stream()), "moe_topk_sigmoid")
    return w, ids


def moe_route_softmax(x, weight, bias, top_k: int):
    """Experts of the ``top_k`` largest ``x @ weight^T + bias`` (fp32), weights the softmax over those."""
    T, E = x.shape[0], weight.shape[0]
    part, splits = _router_logits(x, weight)
    w = torch.empty(T, top_k, dtype=torch.float32, device=x.device)
    ids = torch.empty(T, top_k, dtype=torch.int32, device=x.device)
    _check(load().tgi_moe_topk_logits(_ptr(part), c_int(splits), _ptr(bias), c_int(T), c_int(E), c_int(top_k), _ptr(w), _ptr(ids),
                                      _stream()), "moe_topk_logits")
    return w, ids


def moe_plain_experts(x, w_up, w_down, topk_weights, topk_ids, act: str, gated: bool = False):
    """Experts ``w_up [E, I, H]`` (``gated``: ``[E, 2 I, H]``), ``w_down [E, H, I]`` (``ops.plain_expert_weights``) on their
    routed rows, in bf16 (grouped tcgen05 GEMMs) or fp32; no host synchronisation."""
    lib, st, s = load(), state(x.device), _stream()
    T, H = x.shape
    E, I, Hp = w_up.shape
    up = 2
    if gated:
        I, up = I // 2, 0
    k = topk_ids.shape[1]
    n = T * k
    new = lambda *shape, dtype=x.dtype: torch.empty(*shape, dtype=dtype, device=x.device)
    assert w_up.is_contiguous() and w_down.is_contiguous() and tuple(w_down.shape) == (E, Hp, I) and w_up.dtype == x.dtype
    assert topk_ids.dtype == torch.int32 and topk_weights.dtype == torch.float32
    pos, order, offsets = new(n, dtype=torch.int32), new(n, dtype=torch.int32), new(E + 1, dtype=torch.int32)
    hidden, y, out = new(n, I), new(n, Hp), new(T, Hp)
    if T == 0:
        return x.new_zeros(0, H)
    x = torch.nn.functional.pad(x, (0, Hp - H)) if Hp > H else x.contiguous()
    _check(lib.tgi_moe_sort(_ptr(topk_ids), c_int(n), c_int(0), c_int(E), _ptr(pos), _ptr(order), _ptr(offsets), s), "moe_sort")
    code = c_int(_ACT_CODES[act])
    if x.dtype == torch.float32:
        for mode, src, w, dst in ((up, x, w_up, hidden), (1, hidden, w_down, y)):
            _check(lib.tgi_moe_grouped_f32(c_int(mode), _ptr(src), c_int(n), _ptr(w), c_int(E), c_int(k), c_int(dst.shape[1]),
                                           c_int(w.shape[2]), _ptr(offsets), _ptr(order), code, _ptr(topk_weights), _ptr(dst), s),
                   "moe_grouped_f32")
        _check(lib.tgi_moe_combine_f32(_ptr(y), _ptr(pos), c_int(T), c_int(k), c_int(Hp), _ptr(out), s), "moe_combine_f32")
        return out
    grouped = new(n, Hp)
    _check(lib.tgi_moe_gather(_ptr(x), _ptr(order), _ptr(offsets), c_int(E), c_int(k), c_int(Hp), c_int(n), _ptr(grouped), s),
           "moe_gather")
    for mode, src, w, dst in ((up, grouped, w_up, hidden), (1, hidden, w_down, y)):
        _check(lib.tgi_moe_grouped_gemm(c_int(mode), _ptr(src), c_int(n), _ptr(w), c_int(E), c_int(w.shape[1]), c_int(w.shape[2]),
                                        _ptr(offsets), code, _ptr(topk_weights), _ptr(order), _ptr(dst), c_int(st.sm_count),
                                        _ptr(st.status), s), "moe_grouped_gemm")
    _check(lib.tgi_moe_combine(_ptr(y), _ptr(pos), c_int(T), c_int(k), c_int(Hp), _ptr(out), s), "moe_combine")
    return out if Hp == H else out[:, :H].contiguous()


# ---- multi-adapter LoRA ------------------------------------------------------------------------
def lora_shrink(x: torch.Tensor, a_ptrs: torch.Tensor, ranks: torch.Tensor, token_adapter: torch.Tensor,
                rmax: int) -> torch.Tensor:
    """``v[t] = A_{adapter(t)} x[t]`` in fp32, ``[T, rmax]`` (zero rows for tokens without adapter)."""
    T, H = x.shape
    v = torch.empty(T, rmax, dtype=torch.float32, device=x.device)
    _check(load().tgi_lora_shrink(_ptr(x.contiguous()), _ptr(a_ptrs), _ptr(ranks), _ptr(token_adapter), _ptr(v),
                                  c_int(T), c_int(H), c_int(rmax), _stream()), "lora_shrink")
    return v


def lora_expand(v: torch.Tensor, b_ptrs: torch.Tensor, ranks: torch.Tensor, scales: torch.Tensor,
                token_adapter: torch.Tensor, out: torch.Tensor, col0: int, ncols: int):
    """``out[t, col0:col0+ncols] += scale * B_{adapter(t)} v[t]`` in place (``out`` bf16, rows contiguous)."""
    T, rmax = v.shape
    if out.stride(1) != 1:
        raise KernelError("lora_expand needs unit stride along the columns of `out`")
    _check(load().tgi_lora_expand(_ptr(v), _ptr(b_ptrs), _ptr(ranks), _ptr(scales), _ptr(token_adapter), _ptr(out),
                                  c_ll(out.stride(0)), c_int(col0), c_int(T), c_int(ncols), c_int(rmax), _stream()),
           "lora_expand")
