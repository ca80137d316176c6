"""Loads the native library and declares its C entry points.

There is one execution path: the CUDA kernels of `csrc/`.  If the library cannot be built
or loaded, or no CUDA device is present, the first kernel call raises; nothing falls back
to the CPU or to a library implementation.
"""

from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_longlong, c_void_p

_lib: ctypes.CDLL | None = None
_path: str | None = None
_launches = 0  # kernel launches made through `call` (graph replays are counted by their owner)


class KernelError(RuntimeError):
    """A native entry point refused its arguments or a CUDA call failed."""


_P, _I, _F, _L = c_void_p, c_int, c_float, c_longlong

_SIGNATURES: dict[str, list] = {
    "ns_embed": [_P, _P, _P, _I, _I, _I, _I, _P],
    "ns_take_ids": [_P, _P, _P, _P, _I, _P],
    "ns_add_rmsnorm": [_P, _P, _P, _P, _P, _I, _I, _F, _I, _I, _P],
    "ns_residual_add": [_P, _P, _I, _I, _I, _P],
    "ns_swiglu": [_P, _P, _I, _I, _I, _I, _P],
    "ns_swiglu_rows": [_P, _L, _P, _L, _I, _I, _I, _I, _P],
    "ns_gate_mul_rows": [_P, _L, _P, _L, _I, _I, _I, _F, _F, _F, _I, _P],
    "ns_gemm_f32": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "ns_rope_kv_write": [_P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "ns_attention_generic": [_P, _I, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _F, _I, _I, _I, _F, _I, _P],
    "ns_add_layernorm": [_P, _P, _P, _P, _P, _I, _I, _F, _I, _I, _P],
    "ns_scale_softcap": [_P, _I, _I, _L, _F, _F, _P],
    "ns_qk_norm_rope_store": [_P, _I, _P, _P, _P, _I, _P, _F, _I, _I, _P, _P, _F, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P, _I, _P],
    "ns_delta_prepare": [_P, _I, _P, _I, _P, _P, _P, _L, _L, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _F, _F, _I, _P],
    "ns_rotary_prepare": [_P, _I, _P, _P, _P, _F, _I, _I, _P, _I, _I, _I, _I, _I, _I, _F, _F, _I, _P],
    "ns_linear_scan": [_P, _P, _P, _P, _P, _P, _P, _I, _P, _L, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "ns_ssm_chunked": [_P, _P, _P, _P, _I, _P, _P, _L, _P, _P, _P, _I, _I, _I, _I, _P, _P, _I, _I, _I, _I, _I, _P],
    "ns_ssm_prepare": [_P, _I, _P, _P, _I, _P, _P, _P, _L, _L, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "ns_ssm_gate_norm": [_P, _I, _P, _I, _P, _I, _P, _P, _F, _I, _P, _I, _P, _P, _P, _P, _L, _L, _I, _I, _I, _I, _I, _I, _P],
    "ns_head_norm_gate": [_P, _I, _P, _I, _P, _F, _P, _I, _P, _I, _I, _I, _I, _P],
    "ns_sample_rows": [_P, _L, _I, _I, _P, _P, _P, _P, _P, _P, _P, _P, _P],
    "ns_attention_decode": [_P, _I, _P, _P, _P, _I, _P, _P, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _I, _P],
    "ns_attention_decode_tma": [_P, _I, _P, _P, _L, _P, _I, _P, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _F, _I, _I, _P, _P, _P, _P, _P],
    "ns_gemm_bf16_tc_norm": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P, _I, _I, _F, _P, _P, _P, _P, _I, _P, _P],
    "ns_gemm_bf16_tc_dyt": [_P, _P, _I, _I, _I, _I, _I, _I, _P, _P, _P, _P, _P, _P, _P, _P, _I, _P, _P],
    "ns_rope_token_kernel_from": [_I],
    "ns_gemm_bf16_tc_rope": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P, _I, _I, _F, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I,
                             _P, _P],
    "ns_set_pdl": [_I],
    "ns_full_launch_next": [],
    "ns_attention_decode_stages": [_I],
    "ns_gemm_bf16_tc": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P, _P],
    "ns_gemm_bf16_tc_gated": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P, _P],
    "ns_gemm_bf16_tc_unit": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _F, _F, _F, _P, _P],
    "ns_attention_prefill_tc": [_P, _I, _I, _P, _P, _L, _P, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _F, _I, _P, _P],
    "ns_wait_probe": [_P, _L, _P, _P],
    "ns_attention_decode_kept": [_P, _I, _P, _P, _P, _I, _P, _P, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _I, _I, _I, _F, _I, _I,
                                 _P, _P, _I, _I, _F, _P],
    "ns_attention_prefill_kept": [_P, _I, _P, _P, _P, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _F, _I, _I, _I, _I, _F, _I, _P, _P, _I, _I, _F, _P],
    "ns_attention_generic_sink": [_P, _I, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _F, _I, _I, _I, _F, _P, _P, _I, _I, _F, _I, _P],
    "ns_add_dyt": [_P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P],
    "ns_dyt_join": [_P, _P, _P, _P, _P, _P, _I, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P],
    "ns_head_prepare_store": [_P, _I, _P, _I, _P, _P, _P, _P, _P, _I, _P, _F, _I, _I, _P, _P, _I, _F, _F, _F, _P, _I, _P, _L, _P, _P,
                              _I, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "ns_conv_tail": [_P, _I, _P, _L, _L, _P, _P, _I, _I, _I, _I, _P],
    "ns_attention_prefill": [_P, _I, _P, _P, _P, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _F, _I, _P],
    "ns_stream_mix_norm": [_P, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _F, _I, _I, _P],
    "ns_stream_read": [_P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P],
    "ns_embed_streams": [_P, _P, _P, _I, _I, _I, _F, _I, _I, _P],
    "ns_latent_rope_store": [_P, _I, _P, _P, _P, _I, _P, _F, _I, _P, _F, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "ns_attention_latent": [_P, _L, _L, _P, _L, _L, _P, _P, _I, _P, _P, _P, _P, _L, _P, _L, _L, _I, _I, _I, _I, _I, _F, _I, _I, _P],
    "ns_attention_latent_tc": [_P, _L, _L, _P, _L, _L, _P, _P, _I, _P, _P, _P, _P, _L, _P, _L, _L, _P, _P, _I, _I, _I, _I, _I, _F, _I, _I, _P],
    "ns_cast_f32": [_P, _L, _P, _I, _I, _I, _P],
    "ns_router_logits": [_P, _L, _P, _P, _P, _I, _I, _I, _I, _P],
    "ns_moe_route": [_P, _I, _I, _I, _I, _I, _F, _I, _P, _I, _P, _P, _P],
    "ns_moe_route_plan": [_P, _I, _I, _I, _I, _I, _F, _I, _P, _I, _P, _P, _I, _P, _P, _P, _P],
    "ns_moe_plan": [_P, _I, _I, _P, _P, _P, _P],
    "ns_moe_grouped": [_P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _F, _P],
    "ns_moe_grouped_tc": [_P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _F, _P, _P],
    "ns_moe_pad_rows": [_P, _P, _P, _I, _I, _P],
    "ns_moe_gather": [_P, _P, _P, _I, _I, _I, _I, _P],
    "ns_moe_combine": [_P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P],
    "ns_moe_expert_rows": [_P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _F, _I, _P],
    "ns_activation": [_P, _P, _L, _I, _P, _I, _P],
    "ns_activation_rows": [_P, _L, _P, _L, _I, _I, _I, _P, _I, _P],
    "ns_norm_add": [_P, _P, _P, _P, _P, _I, _I, _F, _I, _P],
    "ns_token_gate": [_P, _L, _P, _L, _P, _I, _I, _P, _I, _I, _I, _P],
    "ns_sigmoid_mul": [_P, _L, _P, _L, _I, _I, _I, _P],
    "ns_add_bias": [_P, _L, _P, _I, _I, _I, _P],
}


def load() -> ctypes.CDLL:
    global _lib, _path
    if _lib is not None:
        return _lib
    from ..csrc.build import ensure_built

    path = ensure_built()
    lib = ctypes.CDLL(str(path))
    lib.ns_last_error.restype = ctypes.c_char_p
    lib.ns_last_error.argtypes = []
    for name, args in _SIGNATURES.items():
        fn = getattr(lib, name, None)
        if fn is None:
            continue  # declared lazily by `declare` when a newer source adds it
        fn.argtypes = args
        fn.restype = c_int
    _lib, _path = lib, str(path)
    return lib


def declare(name: str, argtypes: list) -> None:
    """Adds or replaces the signature of an entry point (used by modules that own a kernel)."""
    _SIGNATURES[name] = argtypes
    if _lib is not None:
        fn = getattr(_lib, name)
        fn.argtypes = argtypes
        fn.restype = c_int


def library_path() -> str | None:
    return _path


def launch_count() -> int:
    return _launches


_timed: list | None = None  # (entry point, start event, end event) of every call while kernel timing is on


def start_kernel_timing() -> None:
    """From now on every entry point's launches are bracketed by CUDA events on the current stream (measurement only:
    the events keep neighbouring kernels from overlapping, and nothing may be captured into a graph meanwhile)."""
    global _timed
    _timed = []


def timing_kernels() -> bool:
    return _timed is not None


def stop_kernel_timing() -> dict[str, tuple[int, float]]:
    """Ends kernel timing: entry point -> (calls, milliseconds on the device in total)."""
    global _timed
    import torch

    rows, _timed = _timed or [], None
    torch.cuda.synchronize()
    out: dict[str, tuple[int, float]] = {}
    for name, a, b in rows:
        n, ms = out.get(name, (0, 0.0))
        out[name] = (n + 1, ms + a.elapsed_time(b))
    return out


def call(name: str, *args) -> None:
    global _launches
    lib = load()
    fn = getattr(lib, name, None)
    if fn is None:
        raise KernelError(f"the native library {_path} has no entry point {name}; rebuild it")
    if _timed is not None:
        import torch

        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        status = fn(*args)
        b.record()
        _timed.append((name, a, b))
    else:
        status = fn(*args)
    _launches += 1
    if status != 0:
        raise KernelError(f"{name} failed with status {status}: {lib.ns_last_error().decode(errors='replace')}")
