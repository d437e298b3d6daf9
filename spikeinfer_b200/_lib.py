"""ctypes binding of ``libspikeinfer_b200.so`` (the C ABI declared in ``include/spikeinfer_b200.h``).

There is no fallback: if the library is missing or a call fails, the operators raise.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import POINTER, Structure, c_char_p, c_float, c_int, c_int32, c_int64, c_uint32, c_void_p
from pathlib import Path

import torch

LIB_PATH = Path(os.environ.get("SPIKEINFER_B200_LIB") or Path(__file__).resolve().parent / "libspikeinfer_b200.so")

# element type codes (include/spikeinfer_b200.h)
F32, BF16, F16, U8, I32 = 0, 1, 2, 3, 4
RESET_SUBTRACT_DELAYED, RESET_HARD_ZERO = 0, 1

STATUS_BAD_BLOCK = 1 << 0
STATUS_BAD_SEQ_LEN = 1 << 1
STATUS_BAD_SLOT = 1 << 2
STATUS_POOL_EXHAUSTED = 1 << 3
STATUS_TABLE_FULL = 1 << 4
STATUS_FREE_LIST_OVERFLOW = 1 << 5
STATUS_ROW_BUSY = 1 << 6
STATUS_DEVICE_WAIT_EXPIRED = 1 << 7
STATUS_BAD_TOKEN = 1 << 8

ROW_FREE, ROW_DECODING, ROW_HELD = 0, 1, 2

MAX_LIF_SITES = 4

ATTN_FORM_AUTO, ATTN_FORM_GENERAL, ATTN_FORM_TCGEN05 = 0, 1, 2

_DTYPE_CODES = {
    torch.float32: F32,
    torch.bfloat16: BF16,
    torch.float16: F16,
    torch.uint8: U8,
    torch.int32: I32,
}


class SpkError(RuntimeError):
    """A C-ABI call returned a non-zero status."""


class LifSite(Structure):
    """Mirror of ``spk_lif_site``."""

    _fields_ = [
        ("x", c_void_p),
        ("x_dtype", c_int32),
        ("H", c_int32),
        ("N", c_int64),
        ("sx_t", c_int64),
        ("sx_tok", c_int64),
        ("sx_h", c_int64),
        ("beta", c_void_p),
        ("threshold", c_void_p),
        ("mem0", c_void_p),
        ("mem_out", c_void_p),
        ("packed", c_void_p),
        ("so_t", c_int64),
        ("so_tok", c_int64),
        ("so_h", c_int64),
        ("slot_mapping", c_void_p),
        ("num_rows", c_int64),
        ("dense", c_void_p),
        ("dense_dtype", c_int32),
        ("_pad", c_int32),
        ("sd_t", c_int64),
        ("sd_tok", c_int64),
        ("sd_h", c_int64),
        ("rope_cos", c_void_p),
        ("rope_sin", c_void_p),
        ("s_rope_tok", c_int64),
        ("mul", c_void_p),
        ("sm_t", c_int64),
        ("sm_tok", c_int64),
        ("sm_h", c_int64),
        ("gated", c_void_p),
        ("sg_t", c_int64),
        ("sg_tok", c_int64),
        ("sg_h", c_int64),
    ]


def _fields(spec: str):
    """ctypes fields from ``"kind name name ...; ..."`` with p = pointer, l = int64, i = int32, f = float."""
    kinds = {"p": c_void_p, "l": c_int64, "i": c_int32, "f": c_float}
    out = []
    for group in spec.split(";"):
        kind, *names = group.split()
        out += [(n, kinds[kind]) for n in names]
    return out


class ResidualNormArgs(Structure):
    """Mirror of ``spk_residual_norm_args``."""

    _fields_ = _fields("p x x_out delta embed ids; l vocab; p w w2 mix prev commit; l state_rows; p positions token_rows "
                       "token_edges active out; l n width; f alpha eps; i dtype delta_dtype; p status")


class QkPrepareArgs(Structure):
    """Mirror of ``spk_qk_prepare_args``."""

    _fields_ = _fields("p q k v; l ld; p q_out k_pool v_pool rot_table positions slot_mapping; l rot_positions n num_blocks; "
                       "i heads kv_heads dim vdim k_pad v_pad k_tiled v_tiled block_size rot_dims unit_norm dtype; f eps _pad; p status")


class SigmoidAttnArgs(Structure):
    """Mirror of ``spk_sigmoid_attn_args``."""

    _fields_ = _fields("p q k_pool v_pool tables seq_lens active tiles head_bias out; l out_stride table_stride table_rows "
                       "max_blocks n num_blocks; p partials; i n_tiles splits heads kv_heads dim vdim k_pad v_pad k_tiled v_tiled block_size dtype; "
                       "f scale out_scale; i overlap; p status")


class DecayAttnArgs(Structure):
    """Mirror of ``spk_decay_attn_args``."""

    _fields_ = _fields("p q k v; l ld; p state; l state_stride state_rows; p decay_pow out active chunks seqs workspace; "
                       "l workspace_bytes n; i n_chunks n_seqs heads dim vdim silu dtype overlap; p status")


class GatedNormArgs(Structure):
    """Mirror of ``spk_gated_norm_args``."""

    _fields_ = _fields("p x w gate; l gate_stride; p out; l out_stride; p partials seq_lens active; l n; i width out_offset splits "
                       "left_width dtype; f eps scale left_scale")


class RmsResidualArgs(Structure):
    """Mirror of ``spk_rms_residual_args``."""

    _fields_ = _fields("p x x_out delta embed ids; l vocab; p pairs pair_slots w1 out1 w2 out2 out2_slots; l pair_rows out2_rows n width; "
                       "i pair_top out2_top out2_tiled dtype delta_dtype; f embed_scale pair_scale eps; p status")


class ExpertRouteArgs(Structure):
    """Mirror of ``spk_expert_route_args``."""

    _fields_ = _fields("p layers ids active slots segs; l n vocab; i n_layers max_experts; p status")


class ExpertsArgs(Structure):
    """Mirror of ``spk_experts_args``."""

    _fields_ = _fields("p x w out segs; l rows pairs; i experts k out_features gated dtype _pad; p status")


class LatentPrepareArgs(Structure):
    """Mirror of ``spk_latent_prepare_args``."""

    _fields_ = _fields("p cq kv; l ld; p w_q w_kv cq_out pool rot_table positions slot_mapping; l rot_positions n num_blocks; "
                       "i q_rank rank rot_dim rank_pad rot_pad tiled block_size dtype; f eps _pad; p status")


class LatentQueryArgs(Structure):
    """Mirror of ``spk_latent_query_args``."""

    _fields_ = _fields("p q w_uk out rot_table positions; l rot_positions n; i heads dim rank rot_dim rank_pad rot_pad dtype _pad; p status")


class LatentAttnArgs(Structure):
    """Mirror of ``spk_latent_attn_args``."""

    _fields_ = _fields("p q pool tables seq_lens active token_rows positions partials stats; l table_stride table_rows max_blocks n num_blocks; "
                       "i splits heads rank rot_dim rank_pad rot_pad tiled block_size dtype overlap; f scale; p status")


class LatentOutArgs(Structure):
    """Mirror of ``spk_latent_out_args``."""

    _fields_ = _fields("p partials stats sink w_uv gate out seq_lens active positions; l gate_stride out_stride n; "
                       "i splits heads vdim rank dtype overlap; p status")


class LatentGatherArgs(Structure):
    """Mirror of ``spk_latent_gather_args``."""

    _fields_ = _fields("p pool tables rows latents rotated; l table_stride table_rows max_blocks num_blocks n_ctx; i n_rows rank_pad block_size _pad; "
                       "p status")


class LatentPrefillArgs(Structure):
    """Mirror of ``spk_latent_prefill_args``."""

    _fields_ = _fields("p q kv kr tiles sink gate out rot_table; l rot_positions n n_ctx gate_stride out_stride; "
                       "i n_tiles heads dim rot_dim vdim dim_pad vdim_pad vec_q vec_out dtype; f scale _pad; p status")


class DeltaArgs(Structure):
    """Mirror of ``spk_delta_args``."""

    _fields_ = _fields("p q k v b a gate; l ld ld2; p conv_q conv_k conv_v a_log dt_bias w_norm state conv_state; l state_rows; "
                       "p positions active out; l out_stride; p chunks portions seqs workspace; l workspace_bytes n; "
                       "i n_chunks n_portions heads kv_heads dim vdim taps dtype; f eps _pad; p status")


# name -> (restype, argtypes); every symbol include/spikeinfer_b200.h declares
I64P = POINTER(c_int64)
SIGNATURES = {
    "spk_version": (c_int, []),
    "spk_last_cuda_error": (c_int, []),
    "spk_error_string": (c_char_p, [c_int]),
    "spk_launch_count": (c_int64, []),
    "spk_nvtx_enabled": (c_int, []),
    "spk_attn_overlap_next_call": (c_int, []),
    "spk_pack": (c_int, [c_void_p, c_int, c_int, I64P, I64P, c_int64, c_void_p, c_void_p]),
    "spk_unpack": (c_int, [c_void_p, c_int64, c_int64, c_void_p, c_int, c_void_p]),
    "spk_lif": (c_int, [c_void_p, c_int, c_int, c_int64, c_int, I64P, I64P, c_int64, c_void_p,
                        c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p]),
    "spk_lif_pack_scatter": (c_int, [POINTER(LifSite), c_int, c_int, c_int64, c_int, c_void_p, c_void_p]),
    "spk_add_rmsnorm": (c_int, [c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_int64, c_int64, c_int, c_void_p]),
    "spk_argmax_workspace_bytes": (c_int64, [c_int64]),
    "spk_argmax": (c_int, [c_void_p, c_int, c_int64, c_int64, c_int64, c_void_p, c_void_p, c_int64, c_void_p]),
    "spk_attn_decode_workspace_bytes": (c_int64, [c_int, c_int64, c_int, c_int, c_int, c_int, c_int64]),
    "spk_attn_decode": (c_int, [
        c_void_p, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_void_p,
        c_void_p, c_int, c_int64, c_int64, c_int64,
        c_int, c_int64, c_int, c_int, c_int, c_int, c_int64, c_int64, c_float,
        c_void_p, c_int64, c_void_p, c_void_p]),
    "spk_attn_decode_static_capacity": (c_int64, []),
    "spk_attn_decode_static": (c_int, [
        c_void_p, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_void_p,
        c_void_p, c_int, c_int64, c_int64, c_int64,
        c_int, c_int64, c_int, c_int, c_int, c_int, c_int64, c_int64, c_float,
        c_void_p, c_void_p]),
    "spk_qk_scores": (c_int, [
        c_void_p, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_int64, c_int64, c_int64,
        c_void_p, c_int64, c_void_p,
        c_void_p, c_int64, c_int, c_int64, c_int, c_int, c_int, c_int, c_int64, c_int64,
        c_void_p, c_void_p]),
    "spk_gather_kv_unpacked": (c_int, [
        c_void_p, c_int64, c_int64, c_int64, c_int64, c_void_p, c_int64, c_int, c_int, c_int, c_int,
        c_int64, c_void_p, c_int, c_void_p, c_void_p]),
    "spk_gather_kv_unpacked_batch": (c_int, [
        c_void_p, c_int64, c_int64, c_int64, c_int64, c_void_p, c_int64, c_int64, c_int64, c_int, c_int, c_int, c_int,
        c_int64, c_void_p, c_int, c_void_p, c_void_p]),
    "spk_meta_init": (c_int, [c_void_p, c_void_p, c_int32, c_void_p, c_void_p, c_void_p, c_void_p,
                              c_void_p, c_void_p, c_int32, c_int32, c_int32, c_int32, c_void_p]),
    "spk_meta_advance": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                 c_void_p, c_void_p, c_int32, c_int32, c_int32, c_int32, c_void_p,
                                 c_void_p]),
    "spk_attn_select_form": (c_int, [c_int]),
    "spk_meta_admit": (c_int, [c_int32, c_void_p, c_int32, c_int64, c_void_p, c_void_p, c_void_p,
                               c_void_p, c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_int32,
                               c_int32, c_void_p, c_void_p]),
    "spk_meta_take": (c_int, [c_void_p, c_void_p, c_int32, c_void_p, c_void_p, c_void_p]),
    "spk_meta_extend": (c_int, [c_int32, c_int32, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                c_void_p, c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_int32, c_int32, c_void_p, c_void_p]),
    "spk_residual_norm": (c_int, [POINTER(ResidualNormArgs), c_void_p]),
    "spk_poly_norm": (c_int, [c_void_p, c_void_p, c_float, c_void_p, c_int64, c_int64, c_int, c_void_p]),
    "spk_qk_prepare": (c_int, [POINTER(QkPrepareArgs), c_void_p]),
    "spk_sigmoid_attn_tile_tokens": (c_int, [c_int] * 6),
    "spk_sigmoid_attn_splits": (c_int, [c_int] * 6 + [c_int64, c_int, c_int, c_int64]),
    "spk_sigmoid_attn": (c_int, [POINTER(SigmoidAttnArgs), c_void_p]),
    "spk_decay_powers": (c_int, []),
    "spk_decay_chunk_tokens": (c_int, [c_int, c_int, c_int, c_int64, c_int]),
    "spk_decay_attn_workspace_bytes": (c_int64, [c_int, c_int, c_int, c_int]),
    "spk_decay_attn_step": (c_int, [POINTER(DecayAttnArgs), c_void_p]),
    "spk_decay_attn_chunks": (c_int, [POINTER(DecayAttnArgs), c_void_p]),
    "spk_gated_norm": (c_int, [POINTER(GatedNormArgs), c_void_p]),
    "spk_rms_residual": (c_int, [POINTER(RmsResidualArgs), c_void_p]),
    "spk_gelu_tanh": (c_int, [c_void_p, c_void_p, c_int64, c_int64, c_int64, c_int, c_void_p]),
    "spk_expert_route": (c_int, [POINTER(ExpertRouteArgs), c_void_p]),
    "spk_expert_rows": (c_int64, [c_int64, c_int, c_int]),
    "spk_experts": (c_int, [POINTER(ExpertsArgs), c_void_p]),
    "spk_latent_prepare": (c_int, [POINTER(LatentPrepareArgs), c_void_p]),
    "spk_latent_query": (c_int, [POINTER(LatentQueryArgs), c_void_p]),
    "spk_latent_attn_splits": (c_int, [c_int] * 7 + [c_int64, c_int, c_int64]),
    "spk_latent_attn": (c_int, [POINTER(LatentAttnArgs), c_void_p]),
    "spk_latent_out": (c_int, [POINTER(LatentOutArgs), c_void_p]),
    "spk_latent_prefill_form": (c_int, [c_int] * 5),
    "spk_latent_gather": (c_int, [POINTER(LatentGatherArgs), c_void_p]),
    "spk_latent_prefill": (c_int, [POINTER(LatentPrefillArgs), c_void_p]),
    "spk_delta_step": (c_int, [POINTER(DeltaArgs), c_void_p]),
    "spk_delta_chunk_tokens": (c_int, [c_int] * 3),
    "spk_delta_workspace_bytes": (c_int64, [c_int, c_int64] + [c_int] * 5),
    "spk_delta_prefill": (c_int, [POINTER(DeltaArgs), c_void_p]),
    "spk_meta_release": (c_int, [c_int32, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                 c_void_p, c_int32, c_int32, c_int32, c_int32, c_int32, c_void_p, c_void_p]),
}

_lib = None
_lib_path = LIB_PATH


def use_library(path: Path) -> None:
    """Load ``path`` (a library of some components, :func:`spikeinfer_b200.build.build_components`) instead of the full
    library.  No effect on a library that is loaded already, provided it is that one or the full one."""
    global _lib_path
    if _lib is not None and _lib_path not in (path, LIB_PATH):
        raise SpkError(f"{_lib_path.name} is loaded already and does not hold what {path.name} holds")
    if _lib is None:
        _lib_path = path


def load() -> ctypes.CDLL:
    """Load the shared library once and declare every entry point's signature."""
    global _lib
    if _lib is not None:
        return _lib
    if not _lib_path.exists():
        raise SpkError(
            f"{_lib_path} is missing: build it with `python -m spikeinfer_b200.build` "
            "(there is no fallback path)"
        )
    lib = ctypes.CDLL(str(_lib_path))
    for name, (restype, argtypes) in SIGNATURES.items():
        try:
            fn = getattr(lib, name)
        except AttributeError:
            if _lib_path == LIB_PATH:
                raise
            continue  # a component this library was built without
        fn.restype = restype
        fn.argtypes = argtypes
    _lib = lib
    return lib


def check(code: int, what: str) -> None:
    if code == 0:
        return
    lib = load()
    msg = lib.spk_error_string(code).decode()
    if code == -100:
        msg += f" [cudaError {lib.spk_last_cuda_error()}]"
    raise SpkError(f"{what}: {msg} ({code})")


def dtype_code(dtype: torch.dtype) -> int:
    try:
        return _DTYPE_CODES[dtype]
    except KeyError:
        raise TypeError(f"{dtype} is not supported by the CUDA kernels") from None


def require_cuda(t: torch.Tensor, name: str) -> None:
    if not t.is_cuda:
        raise SpkError(
            f"{name} is on {t.device}: spikeinfer_b200 operators run on CUDA tensors only "
            "(there is no CPU path)"
        )


def ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def current_stream(device: torch.device) -> int:
    return torch.cuda.current_stream(device).cuda_stream


def i64_array(values) -> ctypes.Array:
    values = list(values)
    return (c_int64 * max(len(values), 1))(*values)
