"""ctypes binding of libplz.so (C ABI in include/plz.h) for torch tensors.

torch is used for device memory and streams only; every computation happens in the library's
sm_100a kernels.  There is no fallback: if the library is missing or a call fails this raises.
"""
from __future__ import annotations

import ctypes as C
import os

import torch

_HERE = os.path.dirname(os.path.abspath(__file__))
_LIB_PATH = os.path.join(_HERE, "libplz.so")
_lib = None


class Weight(C.Structure):
    _fields_ = [("N", C.c_int32), ("K", C.c_int32), ("gs_n", C.c_int32), ("gs_k", C.c_int32),
                ("packed", C.c_void_p), ("packed_pitch", C.c_int64), ("palette", C.c_void_p)]


class Lora(C.Structure):
    _fields_ = [("rank", C.c_int32), ("scale", C.c_float), ("A", C.c_void_p), ("lda", C.c_int64),
                ("B", C.c_void_p), ("ldb", C.c_int64)]


class Logits(C.Structure):
    _fields_ = [("ptr", C.c_void_p), ("dtype", C.c_int32), ("s_n", C.c_int64), ("s_k", C.c_int64),
                ("s_p", C.c_int64)]


class SoftOut(C.Structure):
    _fields_ = [("P", C.c_void_p), ("p_n", C.c_int64), ("p_k", C.c_int64), ("p_p", C.c_int64),
                ("w_soft", C.c_void_p), ("ws_n", C.c_int64), ("ws_k", C.c_int64),
                ("w_hard", C.c_void_p), ("wh_n", C.c_int64), ("wh_k", C.c_int64)]


class Noise(C.Structure):
    _fields_ = [("mode", C.c_int32), ("seed", C.c_uint32), ("ptr", C.c_void_p), ("s_n", C.c_int64),
                ("s_k", C.c_int64), ("s_p", C.c_int64)]


class DeltaPrep(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ldp", C.c_int64), ("off_q", C.c_int32), ("off_k", C.c_int32), ("off_v", C.c_int32), ("off_b", C.c_int32),
                ("a", C.c_void_p), ("lda", C.c_int64), ("taps", C.c_void_p), ("A_log", C.c_void_p), ("dt_bias", C.c_void_p),
                ("conv", C.c_void_p), ("n_taps", C.c_int32), ("B", C.c_int32), ("n", C.c_int32), ("H", C.c_int32), ("G", C.c_int32),
                ("dk", C.c_int32), ("dv", C.c_int32), ("q_scale", C.c_float),
                ("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("logg", C.c_void_p), ("beta", C.c_void_p)]


class DeltaRule(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("logg", C.c_void_p), ("beta", C.c_void_p), ("state", C.c_void_p),
                ("o", C.c_void_p), ("B", C.c_int32), ("n", C.c_int32), ("H", C.c_int32), ("G", C.c_int32), ("dk", C.c_int32), ("dv", C.c_int32)]


class DecayAttn(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("ld", C.c_int64), ("decay", C.c_void_p), ("state", C.c_void_p),
                ("o", C.c_void_p), ("B", C.c_int32), ("n", C.c_int32), ("H", C.c_int32), ("dk", C.c_int32), ("dv", C.c_int32)]


class AttnPrep(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ldp", C.c_int64), ("off_q", C.c_int32), ("off_k", C.c_int32), ("off_v", C.c_int32),
                ("wq", C.c_void_p), ("wk", C.c_void_p), ("mix", C.c_void_p), ("v_first", C.c_void_p), ("v_first_write", C.c_int32),
                ("q", C.c_void_p), ("kc", C.c_void_p), ("vc", C.c_void_p), ("k_batch", C.c_int64), ("v_batch", C.c_int64),
                ("pos", C.c_void_p), ("B", C.c_int32), ("n", C.c_int32), ("qw", C.c_int32), ("kw", C.c_int32), ("vw", C.c_int32),
                ("cap", C.c_int32), ("eps", C.c_float)]


class AttnBias(C.Structure):
    _fields_ = [("q", C.c_void_p), ("ldq", C.c_int64), ("k", C.c_void_p), ("v", C.c_void_p), ("k_batch", C.c_int64), ("v_batch", C.c_int64),
                ("o", C.c_void_p), ("ldo", C.c_int64), ("bias", C.c_void_p), ("ldb", C.c_int64), ("n_bias", C.c_int32), ("bias_top", C.c_void_p),
                ("pos", C.c_void_p), ("host_pos", C.c_int32), ("cap", C.c_int32), ("B", C.c_int32), ("n", C.c_int32), ("H", C.c_int32),
                ("G", C.c_int32), ("dk", C.c_int32), ("dv", C.c_int32), ("sink", C.c_int32), ("scale", C.c_float),
                ("sinks", C.c_void_p), ("k_tok", C.c_int64), ("v_tok", C.c_int64), ("k2", C.c_void_p), ("k2_batch", C.c_int64), ("dk2", C.c_int32),
                ("gate", C.c_void_p), ("ldg", C.c_int64)]


class HeadLinear(C.Structure):
    _fields_ = [("x", C.c_void_p), ("ldx", C.c_int64), ("xh", C.c_int64), ("w", C.c_void_p), ("y", C.c_void_p), ("ldy", C.c_int64), ("yh", C.c_int64),
                ("gate", C.c_void_p), ("ldg", C.c_int64), ("M", C.c_int32), ("H", C.c_int32), ("N", C.c_int32), ("K", C.c_int32)]


class Stream(C.Structure):
    _fields_ = [("y", C.c_void_p), ("ldy", C.c_int64), ("w", C.c_void_p), ("w_offset", C.c_float), ("mult", C.c_float), ("eps", C.c_float),
                ("rows", C.c_int64), ("W", C.c_int32), ("x", C.c_void_p), ("add_rows", C.c_void_p), ("add_vec", C.c_void_p), ("w_next", C.c_void_p),
                ("out", C.c_void_p)]


class LatentPrep(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ldp", C.c_int64), ("off_q", C.c_int32), ("off_c", C.c_int32), ("off_r", C.c_int32), ("wq", C.c_void_p),
                ("wc", C.c_void_p), ("cq", C.c_void_p), ("c", C.c_void_p), ("kr", C.c_void_p), ("c_batch", C.c_int64), ("r_batch", C.c_int64),
                ("pos", C.c_void_p), ("freq", C.c_void_p), ("pairs", C.c_int32), ("m", C.c_float), ("B", C.c_int32), ("n", C.c_int32),
                ("q_rank", C.c_int32), ("R", C.c_int32), ("dr", C.c_int32), ("cap", C.c_int32), ("eps", C.c_float)]


class Rotate(C.Structure):
    _fields_ = [("x", C.c_void_p), ("ldx", C.c_int64), ("xh", C.c_int64), ("out", C.c_void_p), ("ldo", C.c_int64), ("oh", C.c_int64), ("pos", C.c_void_p),
                ("freq", C.c_void_p), ("pairs", C.c_int32), ("m", C.c_float), ("B", C.c_int32), ("n", C.c_int32), ("H", C.c_int32), ("dr", C.c_int32)]


class LatentAttn(C.Structure):
    _fields_ = [("q", C.c_void_p), ("ldq", C.c_int64), ("c", C.c_void_p), ("kr", C.c_void_p), ("c_batch", C.c_int64), ("r_batch", C.c_int64),
                ("o", C.c_void_p), ("ldo", C.c_int64), ("sinks", C.c_void_p), ("pos", C.c_void_p), ("host_pos", C.c_int32), ("cap", C.c_int32),
                ("B", C.c_int32), ("n", C.c_int32), ("H", C.c_int32), ("R", C.c_int32), ("dr", C.c_int32), ("scale", C.c_float)]


_I32, _I64, _P, _F = C.c_int32, C.c_int64, C.c_void_p, C.c_float
_WP, _LP, _GP, _NP = C.POINTER(Weight), C.POINTER(Lora), C.POINTER(Logits), C.POINTER(Noise)

# name -> argtypes; every function returns int32 unless listed in _RESTYPES
SIGNATURES = {
    "plz_version": [],
    "plz_last_error": [],
    "plz_launch_count": [],
    "plz_device_status": [C.POINTER(C.c_uint32)],
    "plz_set_cta_limit": [_I32],
    "plz_set_pair_gemm": [_I32],
    "plz_pack_indices": [_P, _I64, _I64, _I32, _I32, _P, _I64, _P],
    "plz_unpack_indices": [_P, _I64, _I32, _I32, _P, _I64, _I64, _P],
    "plz_dequantize": [_WP, _P, _I64, _I64, _P],
    "plz_hard_fwd": [_WP, _P, _I64, _I32, _LP, _P, _P, _I64, _P],
    "plz_hard_fwd_lora_static": [_WP, _P, _I64, _I32, _LP, _P, _I64, _P],
    "plz_hard_fwd_smallm": [_WP, _P, _I64, _I32, _P, _I64, _P],
    "plz_hard_fwd_smallm_multi": [C.POINTER(_WP), _I32, _P, _I64, _I32, C.POINTER(C.c_void_p), C.POINTER(C.c_int64), _P],
    "plz_set_smallm_overlap": [_I32],
    "plz_soft_select": [_WP, _GP, _NP, _F, _I32, _P, _I64, _I64, _P],
    "plz_dense_fwd": [_P, _I64, _I32, _I32, _P, _I64, _I32, _LP, _P, _P, _I64, _P],
    "plz_bwd_dx": [_WP, _P, _I64, _I32, _LP, _P, _P, _I64, _P],
    "plz_lora_dt": [_LP, _P, _I64, _I32, _I32, _P, _P],
    "plz_bwd_dx_with_dt": [_WP, _P, _I64, _I32, _LP, _P, _P, _I64, _P],
    "plz_dense_bwd_dx": [_P, _I64, _I32, _I32, _P, _I64, _I32, _LP, _P, _P, _I64, _P],
    "plz_bwd_dw_soft": [_WP, _P, _I64, _P, _I64, _I32, _GP, _NP, _F, _P, _P, _P],
    "plz_bwd_dw_soft_lora": [_WP, _P, _I64, _P, _I64, _I32, _GP, _NP, _F, _P, _P, _P, _P, _I32, _P, _P, _P],
    "plz_bwd_dw_soft_scatter": [_WP, _P, _I64, _P, _I64, _I32, _GP, _NP, _F, C.POINTER(C.c_void_p), _I32, _I32, _I32, _P, _P, _P, _I32,
                                _P, _P, _P],
    "plz_peer_alloc": [_I64, C.POINTER(C.c_void_p), C.c_char_p],
    "plz_peer_open": [C.c_char_p, C.POINTER(C.c_void_p)],
    "plz_peer_copy": [_P, _P, _I64, _P],
    "plz_peer_zero": [_P, _I64, _P],
    "plz_peer_close": [_P],
    "plz_peer_free": [_P],
    "plz_reduce_slots": [_P, _I32, _I64, _P, _F, _P],
    "plz_bwd_dw_hard": [_WP, _P, _I64, _P, _I64, _I32, _P, _P],
    "plz_lora_bwd": [_P, _I64, _P, _I64, _P, _P, _I32, _I32, _I32, _I32, _P, _P, _P],
    "plz_rms_rstd": [_P, _I64, _I32, _I32, _F, _P, _P],
    "plz_swiglu_bwd": [_P, _I64, _P, _I64, _P, _I64, _I32, _I32, _P, _I64, _P, _I64, _P],
    "plz_rmsnorm_bwd": [_P, _I64, _P, _I64, _P, _P, _I32, _I32, _P, _I64, _P, _P],
    "plz_hard_fwd_norm": [_WP, _P, _I64, _I32, _P, _P, _P, _I64, _P],
    "plz_mlp_gate_up_fwd": [_WP, _WP, _P, _I64, _I32, _P, _P, _P, _I64, _P],
    "plz_mlp_gate_up_fwd_keep": [_WP, _WP, _P, _I64, _I32, _P, _P, _P, _I64, _P, _P, _I64, _P],
    "plz_adamw_step": [_P, _P, _P, _P, _I32, _F, _I64, _F, _F, _F, _F, _F, _I32, _F, _F, _I32, _P, _I32, _P],
    "plz_hard_fwd_bias": [_WP, _P, _I64, _I32, _P, _P, _I64, _P],
    "plz_col_sum": [_P, _I64, _I32, _I32, _P, _P],
    "plz_soft_weights": [_I32, C.POINTER(_WP), C.POINTER(_GP), C.POINTER(_NP), _F, _I32, C.POINTER(C.POINTER(SoftOut)), _P],
    "plz_soft_bwd_elementwise": [_WP, _P, _I32, _I64, _I64, _P, _I64, _I64, _I64, _GP, _P, _P],
    "plz_weight_grad": [_P, _I64, _P, _I64, _I32, _I32, _I32, _P, _I64, _I64, _P],
    "plz_attn_fwd": [_P, _I64, _P, _I64, _P, _I64, _I32, _I32, _I32, _I32, _I32, _F, _P, _I64, _P, _P],
    "plz_attn_bwd": [_P, _I64, _P, _I64, _P, _I64, _P, _P, _I64, _P, _I32, _I32, _I32, _I32, _I32, _F, _P, _P, _P, _P, _P],
    "plz_attn_decode_ws_bytes": [_I32, _I32, _I32, _I32],
    "plz_attn_decode": [_P, _I64, _P, _P, _I64, _I64, _I32, _I32, _I32, _I32, _I32, _F, _P, _I64, _P, _I64, _P],
    "plz_embed_gather": [_P, _I64, _P, _I64, _I32, _I64, _P, _I64, _P, _P],
    "plz_rmsnorm_fwd": [_P, _I64, _P, _I32, _I32, _F, _P, _I64, _P, _P],
    "plz_add_rmsnorm_fwd": [_P, _I64, _P, _I64, _P, _I64, _P, _I32, _I32, _F, _P, _I64, _P, _P],
    "plz_qknorm_rope_fwd2": [_P, _I64, _P, _I32, _P, _I64, _P, _I64, _P, _I32, _P, _I64, _P, _P, _I64, _I32, _I32, _F, _P],
    "plz_qknorm_rope_fwd": [_P, _I64, _P, _P, _P, _I64, _I32, _I32, _I32, _F, _P, _I64, _P],
    "plz_qknorm_rope_bwd": [_P, _I64, _P, _P, _P, _P, _I64, _I64, _I32, _I32, _I32, _F, _P, _I64, _P, _P],
    "plz_swiglu_fwd": [_P, _I64, _P, _I64, _I32, _I32, _P, _I64, _P],
    "plz_add": [_P, _I64, _P, _I64, _P, _I64, _I32, _I32, _P, _I64, _P],
    "plz_bwd_dw_hard_lora": [_WP, _P, _I64, _P, _I64, _I32, _P, _P, _P, _I32, _P, _P, _P],
    "plz_seq_linear": [_I32, _P, _I64, _I32, _I32, _P, _I64, _I32, _P, _I32, _P, _I64, _I32, _P],
    "plz_head_linear": [_I32, C.POINTER(HeadLinear), _P],
    "plz_seq_embed": [_I32, _P, _I64, _P, _I64, _I32, _I64, _F, _P, _F, _F, _P, _P, _P, _P, _P],
    "plz_seq_stream": [_I32, C.POINTER(Stream), _P],
    "plz_latent_prep": [_I32, C.POINTER(LatentPrep), _P],
    "plz_rotate": [_I32, C.POINTER(Rotate), _P],
    "plz_latent_attn_ws_bytes": [_I32, _I32, _I32, _I32, _I32, _I32, _I32],
    "plz_latent_attn": [_I32, C.POINTER(LatentAttn), _P, _I64, _P],
    "plz_seq_rows_norm": [_I32, _P, _P, _P, _F, _F, _I64, _I32, _P, _P],
    "plz_seq_norm_gate": [_I32, _P, _P, _I64, _P, _F, _I64, _I32, _I32, _P, _P],
    "plz_delta_prep": [_I32, C.POINTER(DeltaPrep), _P],
    "plz_chunk_ws_bytes": [_I32, _I32, _I32, _I32, _I32],
    "plz_delta_rule": [C.POINTER(DeltaRule), _P, _I64, _P],
    "plz_decay_attn": [_I32, C.POINTER(DecayAttn), _P, _I64, _P],
    "plz_attn_prep": [_I32, C.POINTER(AttnPrep), _P],
    "plz_attn_bias_ws_bytes": [_I32, _I32, _I32, _I32, _I32],
    "plz_attn_bias": [_I32, C.POINTER(AttnBias), _P, _I64, _P],
    "plz_advance": [_P, _I32, _P],
    "plz_sample": [_P, _I64, _I32, _I32, _F, _I32, C.c_uint32, _P, _P, _P],
    "plz_distill_loss": [_P, _I64, _P, _I64, _I32, _I32, _F, _F, _F, _P, _P, _P, _I64, _I32, _P],
}
_RESTYPES = {"plz_last_error": C.c_char_p, "plz_launch_count": C.c_uint64, "plz_attn_decode_ws_bytes": C.c_int64,
             "plz_attn_bias_ws_bytes": C.c_int64, "plz_chunk_ws_bytes": C.c_int64, "plz_latent_attn_ws_bytes": C.c_int64}


def lib():
    """Load libplz.so (built by build.py).  Raises if it is absent: there is no other code path."""
    global _lib
    if _lib is None:
        if not os.path.exists(_LIB_PATH):
            raise RuntimeError(f"{_LIB_PATH} is missing: run `python {os.path.join(_HERE, 'build.py')}` first; "
                               "this package has no fallback implementation")
        _lib = C.CDLL(_LIB_PATH)
        for name, args in SIGNATURES.items():
            fn = getattr(_lib, name)
            fn.argtypes = args
            fn.restype = _RESTYPES.get(name, C.c_int32)
    return _lib


class PlzError(RuntimeError):
    pass


def check(rc: int, what: str):
    if rc != 0:
        raise PlzError(f"{what} failed with code {rc}: {lib().plz_last_error().decode()}")


def stream_ptr() -> int:
    return torch.cuda.current_stream().cuda_stream


def device_status():
    """Synchronize and return the device status word (code, where, count); raises if a kernel gave up."""
    out = (C.c_uint32 * 4)()
    check(lib().plz_device_status(out), "plz_device_status")
    return tuple(out)


def _need_cuda(*ts):
    for t in ts:
        if t is not None and not t.is_cuda:
            raise PlzError("libplz works on CUDA tensors only (no CPU path exists)")


def weight_desc(packed: torch.Tensor, palette: torch.Tensor, N: int, K: int, gs_n: int, gs_k: int) -> Weight:
    _need_cuda(packed, palette)
    assert packed.dtype == torch.uint8 and packed.dim() == 2 and packed.stride(1) == 1
    assert palette.dtype == torch.bfloat16 and palette.is_contiguous()
    assert palette.numel() == (N // gs_n) * (K // gs_k) * 4, "palette size does not match the grouping"
    return Weight(N, K, gs_n, gs_k, packed.data_ptr(), packed.stride(0), palette.data_ptr())


def lora_desc(a_rk: torch.Tensor, b_nr: torch.Tensor, scale: float) -> Lora:
    _need_cuda(a_rk, b_nr)
    assert a_rk.dtype == torch.bfloat16 and b_nr.dtype == torch.bfloat16
    assert a_rk.stride(1) == 1 and b_nr.stride(1) == 1 and a_rk.shape[0] == b_nr.shape[1]
    return Lora(a_rk.shape[0], float(scale), a_rk.data_ptr(), a_rk.stride(0), b_nr.data_ptr(), b_nr.stride(0))


def logits_desc(t: torch.Tensor, layout: str) -> Logits:
    """layout 'nk4': tensor [N, K, 4]; layout '4kn': tensor (4, K, N)."""
    _need_cuda(t)
    dt = {torch.float32: 0, torch.float16: 1}[t.dtype]
    if layout == "nk4":
        return Logits(t.data_ptr(), dt, t.stride(0), t.stride(1), t.stride(2))
    return Logits(t.data_ptr(), dt, t.stride(2), t.stride(1), t.stride(0))


def noise_desc(noise, layout: str, seed: int = 0) -> Noise:
    """noise: None (no noise), a fp32 tensor in the given layout, or the string 'hash' (counter-based)."""
    if noise is None:
        return Noise(0, 0, None, 0, 0, 0)
    if isinstance(noise, str):
        return Noise(2, seed & 0xFFFFFFFF, None, 0, 0, 0)
    _need_cuda(noise)
    assert noise.dtype == torch.float32
    if layout == "nk4":
        return Noise(1, 0, noise.data_ptr(), noise.stride(0), noise.stride(1), noise.stride(2))
    return Noise(1, 0, noise.data_ptr(), noise.stride(2), noise.stride(1), noise.stride(0))
