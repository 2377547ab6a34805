"""The compiled kernel libraries and the declaration of their exported functions."""
from __future__ import annotations

import ctypes
import os
from ctypes import c_float, c_int, c_longlong, c_ulonglong, c_void_p

import torch

from ..csrc import build

P, I, F, LL, ULL = c_void_p, c_int, c_float, c_longlong, c_ulonglong

CORE_SOURCES = ("elementwise.cu", "linear_simt.cu", "attention_generic.cu", "sampling.cu", "linear_fused.cu", "gemm_tcgen05.cu")
# Kernels that no model needs unless it is asked for them: the allocation-free entry point and the split-K product it
# is built on (linear_mma.cu), and the two kernels for decode steps of 17 to 64 rows that the library's products with
# this library's small kernels between them still beat (linear_batch.cu: mma.sync with fused prologue and epilogues;
# gemm_splitk.cu: tcgen05 with K cut over a cluster).
EXTRA_SOURCES = ("linear_mma.cu", "linear_batch.cu", "gemm_splitk.cu")
# The kernels of parts that only some designs have (layer norm with the short convolution on a sublayer's input, attention
# whose weights are mixed across heads, the gated recurrence): compiled when a model with such a part is built.
MIXER_SOURCES = ("layernorm_conv.cu", "attention_headmix.cu", "attention_headmix_mma.cu", "attention_headmix_flash.cu",
                 "gated_recurrence.cu")
# The kernels of gated mixers and routed feed-forwards (the linear-attention recurrence, rotation of pairs with unit norm and
# cache write, norms over groups of channels with a gate, sums of normed branches, gated activations, the choice of experts;
# branches that share their first and last product, and residuals of several streams).
GATED_SOURCES = ("linear_attention.cu", "linear_attention_tiles.cu", "gated_ops.cu", "branch_ops.cu")
# The kernels of the state-space mixer (short convolution with silu, the recurrence with a scalar decay, gate then norm) and of
# attention over one low-rank row per position.
STATE_SOURCES = ("state_space.cu", "latent_ops.cu")
# The kernels of sublayers that read the same rows and share their first and last product, of heads with several maps, and of routers
# that read normed rows.
JOINED_SOURCES = ("joined_ops.cu", "attention_diff.cu", "attention_diff_tcgen05.cu")
HEAD_DIM_SOURCES = ("attention_decode.cu", "attention_prefill.cu", "attention_prefill_tcgen05.cu")      # compiled per head size

_SIGNATURES = {
    "pe_embed": [P, I, P, P, I, I, I, F, P],
    "pe_embed_pairs": [P, P, I, P, P, P, P, P, P, LL, P, I, I, I, I, I, I, P],
    "pe_select_tokens": [P, P, P, I, P],
    "pe_rmsnorm": [P, P, P, I, F, P, I, I, I, P],
    "pe_add_rmsnorm": [P, P, I, P, I, F, P, I, I, I, P],
    "pe_swiglu": [P, P, I, I, I, P],
    "pe_residual_add": [P, P, I, LL, P],
    "pe_bias_add": [P, I, P, I, I, I, P],
    "pe_rope_store": [P, I, I, I, I, I, P, P, P, P, P, P, P, I, I, P],
    "pe_linear_simt": [P, I, P, I, P, I, P, I, I, I, I, P],
    "pe_attention_generic": [P, I, P, P, P, I, P, I, P, P, I, I, I, I, I, F, P],
    "pe_argmax": [P, P, I, I, P, P],
    "pe_sample": [P, P, I, I, F, I, F, ULL, P, P, P, P, P],
    "pe_gemm_tcgen05": [P, P, P, I, P, I, I, I, I, I, P, P],
    "pe_gemm_tcgen05_rope": [P, P, P, I, P, I, I, I, I, I, P, P, P, P, P, P, P, I, I, I, P, P],
    "pe_linear_fused": [P, P, P, I, F, P, P, I, P, I, I, I, I, P, P],
    "pe_linear_fused_scaled": [P, P, P, I, F, P, P, I, P, I, F, I, I, I, P, P],
    "pe_norm_gate_up_swiglu": [P, P, I, F, P, P, I, I, I, P, P],
    "pe_gate_up_act": [P, P, P, I, I, I, I, P, P],
    "pe_norm_qkv_rope_store": [P, P, P, I, F, P, P, I, P, I, I, I, I, I, P, P, P, P, P, P, P, I, I, P, P],
    "pe_add_sinusoid": [P, P, P, I, I, P],
    "pe_activation": [P, P, I, I, LL, P],
    "pe_softcap": [P, F, LL, P],
}

_MIXER_SIGNATURES = {
    "pe_layernorm": [P, P, P, I, P, I, F, P, I, I, I, P],
    "pe_layernorm_add": [P, P, I, P, I, P, I, F, I, I, P, I, P, I, F, P, I, P],
    "pe_add_layernorm": [P, P, I, P, I, P, I, P, I, P, I, F, I, I, P, I, P],
    "pe_causal_conv_add": [P, P, I, P, LL, P, P, P, P, I, I, I, I, P],
    "pe_conv_state_update": [P, P, LL, P, P, P, I, I, I, P],
    "pe_dual_layernorm_conv": [P, P, I, P, I, P, I, P, P, P, I, P, I, P, I, P, P, I, LL, P, P, P, P, F, I, I, I, I, I, P],
    "pe_mingru": [P, I, P, LL, P, P, P, P, P, I, I, I, I, P, P],
    "pe_attention_headmix": [P, I, P, P, P, I, P, I, P, P, P, I, I, I, I, I, I, I, I, F, P, I, P, I, I, I, P, P, I, I, I, I, I, P],
    "pe_qknorm_store": [P, I, I, I, I, I, I, P, I, P, I, F, P, P, P, P, P, I, I, P],
    "pe_attention_flashmix": [P, I, P, P, P, P, I, P, P, P, I, I, I, I, I, I, I, F, P, P, I, P, P, I, I, P],
    "pe_attention_headmix_mma": [P, I, P, P, P, P, I, P, P, P, I, I, I, I, I, I, I, I, F, P, P, I, P, P],
}

_GATED_SIGNATURES = {
    "pe_linear_attention": [P, I, I, I, I, I, P, I, I, P, F, F, I, I, P, LL, P, P, P, P, I, I, I, I, I, I, P, P, I, P],
    "pe_rotary_norm_store": [P, I, I, I, I, I, I, I, P, I, I, F, P, P, P, P, P, I, I, P],
    "pe_gated_norm": [P, I, I, I, I, P, I, F, P, I, I, I, P, I, P],
    "pe_normed_sum_add": [P, P, P, P, P, I, P, P, P, P, I, I, I, I, F, F, P],
    "pe_scaled_add": [P, P, I, F, LL, P],
    "pe_add_rows": [P, P, P, I, I, I, P],
    "pe_gated_act": [P, P, I, I, I, I, P, I, I, F, F, P],
    "pe_weighted_act": [P, P, I, I, I, I, P, I, I, P],
    "pe_moe_route": [P, I, I, I, I, P, P, I, I, F, P],
    "pe_moe_route_grouped": [P, I, I, I, P, I, I, I, I, F, P, P, I, P],
    "pe_moe_route_stream_grouped": [P, P, I, P, I, F, P, I, I, I, P, I, I, I, I, F, P, P, I, P],
    "pe_rotary_half_store": [P, I, I, I, I, I, I, I, P, I, F, I, F, P, P, P, P, P, I, I, P, I, P, I, P],
    "pe_moe_route_stream": [P, P, I, F, P, I, I, I, I, P, P, I, I, F, P],
    "pe_heads_prepare": [P, I, I, I, P, P, I, I, I, I, P, P, I, F, P, I, I, P, P, P, I, I, I, I, I, I, P, I, I, F, P, P],
    "pe_gate_heads": [I, P, P, P, P, P, P, P, P, P, P, P, I, P, I, P, I, I, P],
    "pe_stream_mix": [P, LL, LL, P, P, I, P, P, P, P, I, F, P, I, I, I, I, P],
}

_STATE_SIGNATURES = {
    "pe_conv_silu": [P, I, I, I, I, I, P, I, P, I, P, LL, P, P, P, P, P, I, I, P],
    "pe_state_space_scan": [P, I, P, I, I, I, P, I, P, I, P, I, P, LL, P, P, P, P, I, I, I, I, I, I, I, P, P],
    "pe_gate_norm": [P, I, I, I, P, I, I, I, P, I, F, P, P],
    "pe_latent_prepare": [P, I, I, I, I, I, I, I, I, P, I, F, P, I, P, P, P, P, P, P, I, I, I, P, I, P],
    "pe_rmsnorm_cols": [P, I, I, I, I, P, I, F, P, I, P],
    "pe_head_gate": [P, I, P, I, I, I, I, I, P, P],
}

_JOINED_SIGNATURES = {
    "pe_heads_norm_store": [P, I, I, I, I, I, I, I, I, P, I, P, I, F, P, I, P, P, P, P, P, I, I, P],
    "pe_attention_diff_takes": [I, I, I, I],
    "pe_attention_diff": [P, I, P, I, I, P, P, P, I, P, P, P, I, I, I, I, I, I, I, F, F, F, F, I, P],
    "pe_attention_diff_tcgen05_takes": [I, I, I, I],
    "pe_attention_diff_tcgen05": [P, I, P, I, I, P, P, LL, P, I, P, I, I, I, I, I, I, I, F, F, F, F, P, P],
    "pe_map_difference": [P, I, I, I, I, F, F, F, P, I, I, I, P],
    "pe_side_act": [P, I, I, I, I, I, I, I, P, I, I, I, P, I, I, P],
    "pe_route_rows": [P, I, P, I, I, I, I, P, I, I, F, P, P, I, P],
}

_EXTRA_SIGNATURES = {
    "pe_gemm_splitk": [P, P, P, I, P, I, I, I, I, P, P],
    "pe_gemm_splitk_rope": [P, P, P, I, P, I, I, I, I, I, P, P, P, P, P, P, P, I, I, P, P],
    "pe_linear_mma": [P, P, P, I, P, I, I, I, I, P, P, P],
    "pe_linear_mma_splits": [I, I],
    "pe_linear_batch": [P, P, P, I, F, P, P, I, P, I, I, I, I, P, P],
    "pe_batch_norm_gate_up_swiglu": [P, P, I, F, P, P, I, I, I, P, P],
    "pe_batch_norm_qkv_rope_store": [P, P, I, F, P, P, I, P, I, I, I, I, I, P, P, P, P, P, P, P, I, I, P, P],
}

_HEAD_DIM_SIGNATURES = {
    "pe_attention_decode": [P, I, P, P, P, P, I, P, P, I, I, I, I, I, F, I, I, P, P, I, P, P],
    "pe_attention_decode_splits": [I, I, I, I, P],
    "pe_attention_prefill": [P, I, P, P, P, P, I, P, P, P, I, I, I, I, I, F, P],
    "pe_attention_prefill_tcgen05": [P, I, P, P, P, LL, P, I, P, I, I, I, I, I, I, F, I, P, P, P, P],
}

DTYPE_CODE = {torch.float32: 0, torch.bfloat16: 1}


class KernelError(RuntimeError):
    pass


_core = None
_by_head_dim = {}


def declare(lib: ctypes.CDLL, signatures: dict) -> None:
    for name, args in signatures.items():
        fn = getattr(lib, name)
        fn.argtypes = args
        fn.restype = c_int


def core() -> ctypes.CDLL:
    """The library of the kernels every model needs; compiled at the first call."""
    global _core
    if _core is None:
        lib = build.load("core", CORE_SOURCES)
        declare(lib, _SIGNATURES)
        lib.pe_set_pdl(0 if os.environ.get("PICO_ENGINE_PDL", "1") == "0" else 1)
        lib.pe_draw_uniform.argtypes = [ULL, ULL, ULL]
        lib.pe_draw_uniform.restype = c_float
        lib.pe_argmax_scratch_bytes.argtypes = [I, I]
        lib.pe_argmax_scratch_bytes.restype = c_longlong
        lib.pe_sample_scratch_bytes.argtypes = [I, I]
        lib.pe_sample_scratch_bytes.restype = c_longlong
        _core = lib
    return _core


_mixers = None


def mixers() -> ctypes.CDLL:
    """The library of the kernels of layer norm + input convolution, head-mixing attention and the gated recurrence;
    compiled at the first call."""
    global _mixers
    if _mixers is None:
        lib = build.load("mixers", MIXER_SOURCES)
        declare(lib, _MIXER_SIGNATURES)
        lib.pe_set_pdl(0 if os.environ.get("PICO_ENGINE_PDL", "1") == "0" else 1)
        lib.pe_mingru_scratch_floats.argtypes = [I, I, I]
        lib.pe_mingru_scratch_floats.restype = c_longlong
        lib.pe_attention_headmix_tile.argtypes = [I, I, I, I, I, I]
        lib.pe_attention_headmix_tile.restype = c_int
        lib.pe_attention_headmix_scratch_floats.argtypes = [I, I, I, I, I]
        lib.pe_attention_headmix_scratch_floats.restype = c_longlong
        lib.pe_attention_flashmix_group.argtypes = [I, I, I, I]
        lib.pe_attention_flashmix_group.restype = c_int
        lib.pe_attention_flashmix_scratch_floats.argtypes = [I, I, I, I, I, I]
        lib.pe_attention_flashmix_scratch_floats.restype = c_longlong
        lib.pe_attention_headmix_mma_plan.argtypes = [I, I, I, I, ctypes.POINTER(c_int)]
        lib.pe_attention_headmix_mma_plan.restype = c_int
        lib.pe_attention_headmix_mma_scratch_floats.argtypes = [I, I, I, I]
        lib.pe_attention_headmix_mma_scratch_floats.restype = c_longlong
        _mixers = lib
    return _mixers


_gated = None


def gated() -> ctypes.CDLL:
    """The library of the kernels of gated mixers and routed feed-forwards; compiled at the first call."""
    global _gated
    if _gated is None:
        lib = build.load("gated", GATED_SOURCES)
        declare(lib, _GATED_SIGNATURES)
        lib.pe_set_pdl(0 if os.environ.get("PICO_ENGINE_PDL", "1") == "0" else 1)
        lib.pe_linear_attention_scratch_floats.argtypes = [I, I, I, I, I]
        lib.pe_linear_attention_scratch_floats.restype = c_longlong
        _gated = lib
    return _gated


_state = None


def state_space() -> ctypes.CDLL:
    """The library of the kernels of the state-space mixer and of attention over low-rank rows; compiled at the first call."""
    global _state
    if _state is None:
        lib = build.load("state", STATE_SOURCES)
        declare(lib, _STATE_SIGNATURES)
        lib.pe_set_pdl(0 if os.environ.get("PICO_ENGINE_PDL", "1") == "0" else 1)
        lib.pe_state_space_split.argtypes = [I]
        lib.pe_state_space_split.restype = c_int
        lib.pe_state_space_elems.argtypes = [I, I, I]
        lib.pe_state_space_elems.restype = c_longlong
        lib.pe_state_space_scratch_floats.argtypes = [I, I, I, I, I]
        lib.pe_state_space_scratch_floats.restype = c_longlong
        _state = lib
    return _state


_joined = None


def joined() -> ctypes.CDLL:
    """The library of the kernels of sublayers that share their first and last product, of heads with several maps and of routers that
    read normed rows; compiled at the first call."""
    global _joined
    if _joined is None:
        lib = build.load("joined", JOINED_SOURCES)
        declare(lib, _JOINED_SIGNATURES)
        lib.pe_set_pdl(0 if os.environ.get("PICO_ENGINE_PDL", "1") == "0" else 1)
        _joined = lib
    return _joined


_extras = None


def extras() -> ctypes.CDLL:
    """The library of the kernels that are not on a model's default path; compiled at the first call."""
    global _extras
    if _extras is None:
        lib = build.load("extras", EXTRA_SOURCES)
        declare(lib, _EXTRA_SIGNATURES)
        lib.pe_set_pdl(0 if os.environ.get("PICO_ENGINE_PDL", "1") == "0" else 1)
        lib.pe_linear_mma_scratch_bytes.argtypes = [I, I, I]
        lib.pe_linear_mma_scratch_bytes.restype = c_longlong
        _extras = lib
    return _extras


def head_dim_sizes() -> range:
    """The head sizes the tensor-core attention kernels are compiled for on demand."""
    return range(16, 257, 16)


def for_head_dim(head_dim: int) -> ctypes.CDLL:
    """The tensor-core attention kernels compiled for one head size; compiled at the first call."""
    if head_dim not in head_dim_sizes():
        raise KernelError(f"head size {head_dim} is not taken: multiples of 16 from 16 to 256 are")
    lib = _by_head_dim.get(head_dim)
    if lib is None:
        lib = build.load(f"attention_hd{head_dim}", HEAD_DIM_SOURCES, {"PE_HEAD_DIM": str(head_dim)})
        declare(lib, _HEAD_DIM_SIGNATURES)
        lib.pe_set_pdl(0 if os.environ.get("PICO_ENGINE_PDL", "1") == "0" else 1)
        _by_head_dim[head_dim] = lib
    return lib


LAUNCHES = [0]      # kernels of this library launched so far (a captured launch counts once, when it is captured)


def check(code: int, name: str, kernels: int = 1) -> None:
    if code == 0:
        LAUNCHES[0] += kernels
        return
    if code == 10001:
        raise KernelError(f"{name}: sizes or dtypes that this kernel does not take")
    raise KernelError(f"{name}: CUDA error {code} ({torch.cuda.get_device_name() if torch.cuda.is_available() else 'no device'})")


def require_cuda(device) -> torch.device:
    device = torch.device(device)
    if device.type != "cuda":
        raise KernelError(f"this library computes on CUDA devices only, not on {device}")
    if not torch.cuda.is_available():
        raise KernelError("no CUDA device is available, and this library has no CPU implementation")
    return device


def stream_ptr() -> int:
    """The raw handle of torch's current CUDA stream (the quick way: no Stream object is made)."""
    return torch._C._cuda_getCurrentRawStream(torch.cuda.current_device())
