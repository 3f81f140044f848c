"""ctypes binding of libcdeep.so (include/cdeep.h).

There is no fallback: if the library is missing the import of any accelerated module
raises, and every non-zero status code becomes a Python exception.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import c_char_p, c_float, c_int, c_longlong, c_size_t, c_void_p

LIB_PATH = os.path.join(os.path.dirname(os.path.abspath(__file__)), "libcdeep.so")
CHECKS_LIB_PATH = os.path.join(os.path.dirname(os.path.abspath(__file__)), "libcdeep_checks.so")

ABI_VERSION = 4



class WindowAttn(ctypes.Structure):
    """cd_window_attn of include/cdeep.h."""
    _fields_ = ([(n, c_void_p) for n in ("q", "k", "v")] + [("ldp", c_longlong)]
                + [(n, c_void_p) for n in ("q_w", "k_w", "r1", "r2", "talk", "ring_k", "ring_v", "out")]
                + [("ldo", c_longlong), ("pos_dev", c_void_p)]
                + [(n, c_float) for n in ("scale", "eps", "out_scale")]
                + [(n, c_int) for n in ("B", "S", "H", "G", "dim", "dp", "vdim", "vp", "window", "keep",
                                        "pos0", "normed")])


class LinearAttn(ctypes.Structure):
    """cd_linear_attn of include/cdeep.h."""
    _fields_ = ([(n, c_void_p) for n in ("q", "k", "v", "gate", "inner")] + [("ldp", c_longlong)]
                + [(n, c_void_p) for n in ("a2", "a2_b", "norm_w", "state", "out")]
                + [("ldo", c_longlong), ("log_decay", c_void_p), ("o_raw", c_void_p)]
                + [(n, c_float) for n in ("inv_tau", "eps", "out_scale", "q_scale")]
                + [(n, c_int) for n in ("B", "S", "H", "dk", "dkp", "dv", "dvp", "rank")])


class LatentAttn(ctypes.Structure):
    """cd_latent_attn of include/cdeep.h."""
    _fields_ = ([(n, c_void_p) for n in ("q", "kv", "gate")] + [("ldp", c_longlong)]
                + [(n, c_void_p) for n in ("norm_w", "cos_t", "sin_t", "uk", "uk_t", "uv", "cache", "out")]
                + [("ldo", c_longlong), ("pos_dev", c_void_p)]
                + [(n, c_float) for n in ("scale", "eps", "out_scale")]
                + [(n, c_int) for n in ("B", "S", "H", "dim", "dimp", "rot", "rotp", "rank", "rankp", "vdim", "vp",
                                        "capacity", "positions", "pos0")])


class DeltaAttn(ctypes.Structure):
    """cd_delta_attn of include/cdeep.h."""
    _fields_ = ([(n, c_void_p) for n in ("q", "k", "v", "b")] + [("ldp", c_longlong), ("zg", c_void_p),
                                                                 ("ldz", c_longlong)]
                + [(n, c_void_p) for n in ("taps_w", "rate", "dt_bias", "norm_w", "ring", "state", "out")]
                + [("ldo", c_longlong)] + [(n, c_void_p) for n in ("act", "inv", "o_raw", "pos_dev")]
                + [(n, c_float) for n in ("eps", "out_scale")]
                + [(n, c_int) for n in ("B", "S", "H", "G", "dk", "dkp", "dv", "dvp", "taps", "pos0")])


_WINDOW_FN = (c_int, [ctypes.POINTER(WindowAttn), c_int, c_void_p])
_LATENT_FN = (c_int, [ctypes.POINTER(LatentAttn), c_int, c_void_p])
_DELTA_FN = (c_int, [ctypes.POINTER(DeltaAttn), c_int, c_void_p])
_GLA_FN = (c_int, [ctypes.POINTER(LinearAttn), c_int, c_void_p])

# name -> (restype, argtypes); mirrors include/cdeep.h one to one
SIGNATURES = {
    "cd_version": (c_int, []),
    "cd_error_string": (c_char_p, [c_int]),
    "cd_last_cuda_error": (c_char_p, []),
    "cd_max_groups": (c_int, []),
    "cd_checks_enabled": (c_int, []),
    "cd_splitk_workspace_bytes": (c_size_t, []),
    "cd_splitk_workspace_set": (c_int, [c_void_p, c_size_t, c_void_p]),
    "cd_splitk_ranges": (c_int, [c_int, c_int, c_int]),
    "cd_splitk_config": (c_int, [c_int]),
    "cd_status_fetch": (c_int, [ctypes.POINTER(c_int)]),
    "cd_selftest_wait_timeout": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_void_p]),
    "cd_route_workspace_bytes": (c_size_t, [c_int, c_int]),
    "cd_route": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p,
                         c_void_p, c_void_p, c_void_p, c_size_t, c_void_p]),
    "cd_route_static_max_tokens": (c_int, [c_int]),
    "cd_route_static": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p,
                                c_void_p, c_void_p, c_void_p, c_void_p]),
    "cd_rmsnorm": (c_int, [c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_void_p, c_void_p,
                           c_int, c_int, c_void_p]),
    "cd_rmsnorm_split": (c_int, [c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_void_p, c_int,
                                 c_int, c_void_p]),
    "cd_gather_rows": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p]),
    "cd_qk_norm_rope": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_float, c_int,
                                c_int, c_int, c_int, c_int, c_int, c_void_p]),
    "cd_decode_rope_append": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_float,
                                      c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_longlong,
                                      c_longlong, c_longlong, c_int, c_void_p, c_void_p]),
    "cd_decode_attention_workspace_bytes": (c_size_t, [c_int, c_int, c_int, c_int, c_int]),
    "cd_decode_attention": (c_int, [c_void_p, c_longlong, c_void_p, c_void_p, c_longlong,
                                    c_longlong, c_longlong, c_void_p, c_longlong, c_float, c_int,
                                    c_int, c_int, c_int, c_void_p, c_int, c_void_p, c_void_p,
                                    c_size_t, c_void_p]),
    "cd_attention_prefill_supported": (c_int, [c_int, c_int, c_int, c_int, c_int]),
    "cd_attention_prefill": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_float,
                                     c_void_p]),
    "cd_gate_up_packed_rows": (c_int, [c_int, c_int]),
    "cd_moe_up": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int,
                          c_int, c_void_p]),
    "cd_moe_up_pair": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p,
                               c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
    "cd_pack_gate_up": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                c_void_p]),
    "cd_pack_down": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "cd_moe_down": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int,
                            c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int,
                            c_void_p]),
    "cd_peer_put_i32": (c_int, [c_void_p, c_int, c_void_p, c_int, c_longlong, c_void_p]),
    "cd_ep_plan": (c_int, [c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_longlong, c_int, c_void_p,
                           c_void_p, c_void_p, c_void_p]),
    "cd_push_rows": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p, c_int,
                             c_int, c_void_p]),
    "cd_peer_barrier": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "cd_moe_down_push": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                 c_int, c_void_p]),
    "cd_moe_combine": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                               c_void_p, c_void_p, c_int, c_int, c_void_p]),
    "cd_mu_qkv": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                          c_void_p]),
    "cd_mu_qkv_rope_supported": (c_int, [c_int, c_int, c_int, c_int, c_int]),
    "cd_mu_qkv_rope": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                               c_void_p, c_void_p, c_void_p, c_void_p, c_float, c_int, c_int,
                               c_int, c_int, c_int, c_void_p]),
    "cd_mu_proj": (c_int, [c_void_p, c_void_p, c_void_p, c_float, c_float, c_int, c_float, c_float,
                           c_void_p, c_int, c_int, c_void_p]),
    "cd_linear": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int,
                          c_int, c_int, c_void_p]),
    "cd_embed_rows": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p]),
    "cd_rmsnorm_f32": (c_int, [c_void_p, c_void_p, c_float, c_float, c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
    "cd_embed_positions": (c_int, [c_void_p] * 4 + [c_int] * 5 + [c_void_p] + [c_int] * 4 + [c_void_p]),
    "cd_layernorm_f32": (c_int, [c_void_p, c_void_p, c_float, c_void_p, c_int, c_int, c_int, c_int, c_void_p]),
    "cd_linear_f32out": (c_int, [c_void_p, c_longlong, c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_int, c_int,
                                 c_int, c_void_p]),
    "cd_project": (c_int, [c_void_p, c_longlong, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_void_p]),
    "cd_linear_f32": (c_int, [c_void_p, c_longlong, c_void_p, c_void_p, c_void_p, c_float, c_int, c_void_p, c_void_p,
                              c_int, c_int, c_int, c_int, c_void_p]),
    "cd_glu_up": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_float, c_float,
                          c_float, c_void_p]),
    "cd_glu_f32": (c_int, [c_void_p, c_void_p, c_int, c_int, c_float, c_float, c_float, c_void_p]),
    "cd_window_attention_supported": (c_int, [ctypes.POINTER(WindowAttn)]),
    "cd_window_attention_norm": _WINDOW_FN,
    "cd_window_attention_rows": _WINDOW_FN,
    "cd_window_attention_decode_workspace_bytes": (c_size_t, [ctypes.POINTER(WindowAttn)]),
    "cd_window_attention_decode": (c_int, [ctypes.POINTER(WindowAttn), c_void_p, c_size_t, c_int, c_void_p]),
    "cd_window_attention_prefill_supported": (c_int, [ctypes.POINTER(WindowAttn)]),
    "cd_window_attention_prefill": (c_int, [ctypes.POINTER(WindowAttn), c_void_p]),
    "cd_window_attention_append": _WINDOW_FN,
    "cd_gla_supported": (c_int, [ctypes.POINTER(LinearAttn)]),
    "cd_gla_step": _GLA_FN,
    "cd_gla_decay": _GLA_FN,
    "cd_gla_sequence": _GLA_FN,
    "cd_gla_finish": _GLA_FN,
    "cd_gla_chunk_workspace_bytes": (c_size_t, [ctypes.POINTER(LinearAttn)]),
    "cd_latent_prepare": _LATENT_FN,
    "cd_latent_rows": _LATENT_FN,
    "cd_latent_decode_workspace_bytes": (c_size_t, [ctypes.POINTER(LatentAttn)]),
    "cd_latent_decode": (c_int, [ctypes.POINTER(LatentAttn), c_void_p, c_size_t, c_void_p]),
    "cd_latent_prefill_supported": (c_int, [ctypes.POINTER(LatentAttn)]),
    "cd_latent_prefill": (c_int, [ctypes.POINTER(LatentAttn), c_void_p, c_void_p]),
    "cd_delta_supported": (c_int, [ctypes.POINTER(DeltaAttn)]),
    "cd_delta_prepare": _DELTA_FN,
    "cd_delta_sequence": _DELTA_FN,
    "cd_delta_finish": _DELTA_FN,
    "cd_delta_step_supported": (c_int, [ctypes.POINTER(DeltaAttn)]),
    "cd_delta_step": _DELTA_FN,
    "cd_delta_chunk_workspace_bytes": (c_size_t, [ctypes.POINTER(DeltaAttn)]),
    "cd_delta_chunk": (c_int, [ctypes.POINTER(DeltaAttn), c_void_p, c_size_t, c_void_p]),
    "cd_route_top": (c_int, [c_void_p, c_longlong, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p]),
    "cd_gather_div": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_longlong, c_int, c_int, c_void_p]),
    "cd_combine_top": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_float, c_void_p, c_int, c_int, c_int, c_void_p]),
    "cd_gla_chunk": (c_int, [ctypes.POINTER(LinearAttn), c_void_p, c_size_t, c_void_p]),
}

_lib = None


class CdeepError(RuntimeError):
    """A libcdeep entry point returned a non-zero status."""


def open_library(path: str) -> ctypes.CDLL:
    """Opens one build of the library and binds every declared entry point."""
    if not os.path.exists(path):
        raise ImportError(
            f"{path} is missing: build it with `python -m complexity_deep_b200.build` "
            "(nvcc, sm_100a). There is no CPU or PyTorch fallback for these kernels.")
    lib = ctypes.CDLL(path)
    for name, (res, args) in SIGNATURES.items():
        fn = getattr(lib, name)  # AttributeError if a declared symbol is not exported
        fn.restype = res
        fn.argtypes = args
    if lib.cd_version() != ABI_VERSION:
        raise ImportError(f"libcdeep ABI {lib.cd_version()} != expected {ABI_VERSION}; rebuild")
    return lib


def load() -> ctypes.CDLL:
    """Loads the library once; raises when it is missing or its ABI version differs.
    CDEEP_CHECKS=1 in the environment selects the checking build (libcdeep_checks.so)."""
    global _lib
    if _lib is None:
        _lib = open_library(CHECKS_LIB_PATH if os.environ.get("CDEEP_CHECKS") == "1" else LIB_PATH)
    return _lib


def check(status: int, what: str) -> None:
    if status != 0:
        lib = load()
        msg = lib.cd_error_string(status).decode()
        detail = lib.cd_last_cuda_error().decode() if status in (2, 3) else ""
        raise CdeepError(f"{what}: {msg}" + (f" ({detail})" if detail else ""))
