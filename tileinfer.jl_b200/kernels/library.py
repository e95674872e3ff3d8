"""Loads the compiled kernel library and declares its C entry points.

There is no fallback: if the library cannot be built or loaded, importing the kernels
raises with the reason.
"""
from __future__ import annotations

import ctypes
from ctypes import c_char_p, c_float, c_int, c_longlong, c_uint, c_void_p

from . import build as _build

_lib = None
# Number of kernels launched through this module so far (a launch inside a CUDA-graph capture counts
# once; its replays are counted by whoever replays the graph).
launch_count = 0
pinned_stream = None          # the stream handle for the launches of a forward pass (see ``stream_scope``)
call_counts = {}              # entry point -> calls that launched (tests read which kernels a step used)


class _Counted:
    """A C entry point that launches ``kernels`` kernels per call; a call that refuses its sizes
    (return code 2) has launched none."""
    __slots__ = ("fn", "kernels", "name")

    def __init__(self, fn, name, kernels=1):
        self.fn, self.name, self.kernels = fn, name, kernels

    def __call__(self, *args):
        global launch_count
        rc = self.fn(*args)
        if rc != 2:
            launch_count += self.kernels
            call_counts[self.name] = call_counts.get(self.name, 0) + 1
        return rc


def current_stream() -> int:
    """The CUDA stream the next launch goes to: the one pinned for the running forward pass, else torch's
    current stream (looking that up costs more than a launch, so a pass looks it up once)."""
    if pinned_stream is not None:
        return pinned_stream
    import torch
    return torch.cuda.current_stream().cuda_stream


class stream_scope:
    """Pins torch's current stream for the launches made inside (a forward pass makes hundreds)."""

    def __enter__(self):
        global pinned_stream
        import torch
        self.before = pinned_stream
        pinned_stream = torch.cuda.current_stream().cuda_stream
        return self

    def __exit__(self, *exc):
        global pinned_stream
        pinned_stream = self.before
        return False


def add_launches(n: int) -> None:
    global launch_count
    launch_count += n


class KernelError(RuntimeError):
    pass


_P, _I, _L, _F, _U = c_void_p, c_int, c_longlong, c_float, c_uint
_SIGNATURES = {
    "ti_embed": [_P, _P, _P, _I, _I, _I, _I, _P, _P],
    "ti_gather_rows": [_P, _P, _P, _I, _I, _I, _P],
    "ti_xielu": [_P, _P, _L, _F, _F, _F, _F, _I, _P],
    "ti_rmsnorm": [_P, _P, _P, _I, _I, _F, _I, _P],
    "ti_add_rmsnorm": [_P, _P, _P, _I, _L, _P, _P, _I, _I, _F, _I, _P],
    "ti_add": [_P, _P, _L, _I, _P],
    "ti_attention_inputs": [_P, _L, _P, _I, _L, _P, _P, _P, _P, _P, _F, _P, _I, _I, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P],
    "ti_attention_plain": [_P, _P, _P, _P, _P, _I, _P, _P, _F, _I, _I, _I, _I, _I, _I, _P, _I, _P],
    "ti_attention_plain_biased": [_P, _P, _P, _P, _P, _I, _P, _P, _F, _I, _I, _I, _I, _I, _I, _P, _I, _P, _I, _I, _P],
    "ti_attention_plain_ruled": [_P, _P, _P, _P, _P, _I, _P, _P, _F, _I, _I, _I, _I, _I, _I, _P, _I, _P, _I, _F, _P, _I, _P],
    "ti_attention_plain_kept": [_P, _P, _P, _P, _P, _I, _P, _P, _F, _I, _I, _I, _I, _I, _I, _P, _I, _P, _I, _F, _P, _I, _I, _P],
    "ti_gemm_plain": [_P, _L, _P, _L, _P, _I, _I, _I, _I, _F, _F, _F, _F, _I, _P],
    "ti_argmax": [_P, _L, _I, _I, _P, _P, _P, _P, _P, _P],
    "ti_sample": [_P, _L, _I, _I, _F, _I, _F, _P, _P, _P, _P, _P],
    "ti_sample_shared": [_P, _L, _I, _I, _F, _I, _F, _P, _P, _P, _P, _I, _P],
    "ti_random_normal": [_P, _I, _L, _L, _U, _U, _F, _F, _P],
    "ti_wait_probe": [_P, _I, _I, _P, _P],
}


_KERNELS_PER_CALL = {"ti_memory_chunks": 3, "ti_ssm_chunks": 3, "ti_ssm_chunks_tc": 3}


def lib():
    """The loaded library (built at the first call if the sources changed)."""
    global _lib
    if _lib is not None:
        return _lib
    try:
        path = _build.build()
        handle = ctypes.CDLL(path)
    except Exception as e:                      # BuildError, OSError
        raise KernelError(f"tileinfer_b200 cannot run without its CUDA kernel library: {e}") from e
    handle.ti_last_error.restype = c_char_p
    handle.ti_last_error.argtypes = []
    handle.ti_sampling_uniform.restype = c_float
    handle.ti_sampling_uniform.argtypes = [_U, _U]
    handle.ti_argmax_chunks.restype = c_int
    handle.ti_argmax_chunks.argtypes = [c_int]
    handle.ti_gemm_tcgen05_decode_plan.restype = c_int
    handle.ti_gemm_tcgen05_decode_plan.argtypes = [c_int] * 5 + [ctypes.POINTER(c_int)] * 2
    class _Lib:
        pass
    wrapped = _Lib()
    wrapped.ti_last_error = handle.ti_last_error
    wrapped.ti_sampling_uniform = handle.ti_sampling_uniform
    wrapped.ti_argmax_chunks = handle.ti_argmax_chunks
    wrapped.ti_gemm_tcgen05_decode_plan = handle.ti_gemm_tcgen05_decode_plan
    handle.ti_expert_plan_max_tiles.restype, handle.ti_expert_plan_max_tiles.argtypes = c_int, [c_int, c_int, c_int]
    wrapped.ti_expert_plan_max_tiles = handle.ti_expert_plan_max_tiles
    handle.ti_memory_chunk_pitch.restype, handle.ti_memory_chunk_pitch.argtypes = c_int, [c_int, c_int]
    wrapped.ti_memory_chunk_pitch = handle.ti_memory_chunk_pitch
    wrapped.handle = handle
    for name, args in _SIGNATURES.items():
        fn = getattr(handle, name)
        fn.restype = c_int
        fn.argtypes = args
        setattr(wrapped, name, _Counted(fn, name, _KERNELS_PER_CALL.get(name, 1)))
    _lib = wrapped
    return wrapped


def set_pdl(enabled: bool) -> None:
    """Launch kernels as programmatic dependents of their predecessors (default) or strictly one
    after the other."""
    h = lib().handle
    h.ti_set_pdl.restype = None
    h.ti_set_pdl.argtypes = [c_int]
    h.ti_set_pdl(1 if enabled else 0)


def declare(name: str, argtypes, restype=c_int):
    """Declare one more entry point (used by kernel files added later)."""
    fn = getattr(lib().handle, name)
    fn.restype = restype
    fn.argtypes = argtypes
    return fn


def check(rc: int, what: str) -> None:
    if rc != 0:
        raise KernelError(f"{what}: {lib().ti_last_error().decode()}")

_SIGNATURES_FAST = {
    "ti_gemv_bf16": [_P, _L, _P, _L, _P, _I, _I, _I, _I, _I, _F, _F, _F, _F, _P],
    "ti_gemm_tcgen05": [_P, _L, _P, _L, _P, _I, _I, _I, _I, _I, _F, _F, _F, _F, _P, _P],
    "ti_gemm_tcgen05_decode": [_P, _L, _P, _L, _P, _I, _I, _I, _I, _I, _I, _F, _F, _F, _F, _P, _P],
    "ti_attention_prefill": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _F, _I, _I, _I, _I, _I, _P],
    "ti_attention_decode": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _P, _F, _I, _I, _I, _I, _I, _I, _I, _P],
    "ti_attention_decode_shared": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _P, _P, _P, _F, _I, _I, _I, _I, _I, _I, _I, _P],
    "ti_attention_prefill_tc": [_P, _P, _P, _P, _I, _P, _I, _P, _P, _P, _I, _I, _I, _F, _I, _I, _I, _I, _I, _P, _P],
}
# The same kernels with a sink: a last argument [heads] float32 (or null) before the stream.
_SIGNATURES_FAST["ti_attention_prefill_sink"] = _SIGNATURES_FAST["ti_attention_prefill"][:-1] + [_P, _P]
_SIGNATURES_FAST["ti_attention_decode_sink"] = _SIGNATURES_FAST["ti_attention_decode_shared"][:-1] + [_P, _P]
# ... and with a chunk, a bias table by distance and its length after the sink
_SIGNATURES_FAST["ti_attention_prefill_biased"] = _SIGNATURES_FAST["ti_attention_prefill"][:-1] + [_P, _I, _P, _I, _P]
_SIGNATURES_FAST["ti_attention_prefill_tc_biased"] = _SIGNATURES_FAST["ti_attention_prefill_tc"][:-1] + [_P, _I, _P, _I, _P]
_SIGNATURES_FAST["ti_attention_decode_biased"] = _SIGNATURES_FAST["ti_attention_decode_shared"][:-1] + [_P, _I, _P, _I, _P]
# ... and with a cap of the scores and a slope per head after those
for _name in ("prefill", "prefill_tc", "decode"):
    _SIGNATURES_FAST[f"ti_attention_{_name}_ruled"] = _SIGNATURES_FAST[f"ti_attention_{_name}_biased"][:-1] + [_F, _P, _P]
    # ... and with a number of first positions that stay visible beside the window
    _SIGNATURES_FAST[f"ti_attention_{_name}_kept"] = _SIGNATURES_FAST[f"ti_attention_{_name}_ruled"][:-1] + [_I, _P]
_SIGNATURES_FAST["ti_attention_prefill_tc_sink"] = _SIGNATURES_FAST["ti_attention_prefill_tc"][:-1] + [_P, _P]
_SIGNATURES.update(_SIGNATURES_FAST)

# The 32-bit residual stream, latent attention's inputs, per-head and per-expert products, activations.
_SIGNATURES.update({
    "ti_embed_positions32": [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P, _P],
    "ti_cast_rows": [_P, _P, _L, _I, _P],
    "ti_norm32": [_P, _P, _I, _P, _I, _I, _F, _I, _I, _P],
    "ti_branch_norm_add32": [_P, _P, _P, _I, _L, _P, _I, _P, _P, _I, _F, _F, _P, _P, _I, _F, _I, _I, _I, _P],
    "ti_latent_inputs": [_P, _L, _P, _I, _L, _P, _P, _P, _P, _F, _P, _I, _I, _I, _I, _P, _I, _P, _I, _L, _I, _P],
    "ti_head_gemm": [_P, _L, _P, _L, _P, _I, _I, _I, _I, _I, _P],
    "ti_gelu": [_P, _P, _L, _I, _I, _P],
    "ti_gated_token_embedding": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "ti_gated_unit_limit": [_P, _P, _I, _I, _F, _P, _I, _P, _F, _F, _I, _P],
    "ti_router_topk": [_P, _P, _P, _I, _I, _I, _I, _I, _P, _P, _I, _P],
    "ti_expert_plan": [_P, _I, _I, _I, _I, _P, _P, _P, _P],
    "ti_expert_gather": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
    "ti_grouped_gemm": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _P, _F, _F, _I, _P],
    "ti_gemm_tcgen05_grouped": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _P, _P],
    "ti_gemm_tcgen05_heads": [_P, _P, _P, _I, _I, _I, _I, _P, _P],
    "ti_expert_combine": [_P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
})

# A state carried from token to token (linear attention with decay), projections through a short convolution, two sublayers
# added at once, routers with more rules, unclamped gated units.
_SIGNATURES.update({
    "ti_lightning_scan": [_P, _P, _L, _I, _I, _I, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P],
    "ti_lightning_out": [_P, _P, _P, _L, _P, _F, _I, _I, _I, _P],
    "ti_conv_attention_inputs": [_P, _L, _P, _P, _I, _P, _P, _P, _F, _P, _I, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I,
                                 _I, _I, _I, _I, _I, _P],
    "ti_conv_state_update": [_P, _P, _L, _P, _I, _P, _P, _I, _I, _I, _P],
    "ti_sigmoid_gate": [_P, _P, _P, _L, _I, _I, _I, _I, _I, _I, _P],
    "ti_sum_add_norm32": [_P, _P, _P, _I, _L, _P, _P, _I, _L, _P, _P, _I, _F, _I, _I, _I, _P],
    "ti_router_select": [_P, _P, _P, _L, _I, _I, _I, _I, _I, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P, _P, _P, _I, _P],
    "ti_gated_act": [_P, _P, _I, _I, _I, _I, _P],
})

# A scaled embedding plus a row chosen by a hash of two consecutive tokens, rows cast into a wider buffer, a rotation of a part of
# every head in place.
_SIGNATURES.update({
    "ti_embed_bigram32": [_P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _F, _L, _L, _L, _I, _P, _P],
    "ti_last_token_update": [_P, _P, _P, _P, _I, _P],
    "ti_cast_rows_ld": [_P, _L, _P, _I, _I, _I, _P],
    "ti_rotate_heads": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P],
})

# Several copies of the residual stream; recurrences over a matrix state with decays that depend on the token; their inputs and outputs.
_SIGNATURES.update({
    "ti_streams_begin": [_P, _P, _I, _I, _I, _P],
    "ti_streams_read_norm": [_P, _P, _P, _I, _P, _P, _F, _I, _I, _I, _I, _P],
    "ti_streams_update": [_P, _P, _P, _I, _L, _P, _P, _P, _I, _P, _P, _P, _F, _I, _I, _I, _I, _P],
    "ti_decay_scan": [_P, _P, _L, _I, _I, _I, _P, _P, _P, _P, _L, _P, _P, _I, _I, _I, _I, _I, _P],
    "ti_delta_scan": [_P, _P, _L, _P, _P, _P, _P, _L, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "ti_shift_blend": [_P, _P, _P, _I, _P, _L, _P, _P, _I, _I, _I, _I, _P],
    "ti_delta_inputs": [_P, _P, _L, _P, _I, _P, _L, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P],
    "ti_history_update": [_P, _L, _P, _L, _I, _P, _P, _I, _I, _I, _P],
    "ti_heads_norm_gate": [_P, _P, _P, _L, _P, _I, _F, _P, _P, _P, _P, _L, _P, _I, _I, _I, _I, _I, _P],
    "ti_pair_combine": [_P, _P, _P, _I, _L, _P, _P, _I, _L, _P, _P, _I, _F, _F, _F, _I, _I, _I, _P],
})

# Gated additions to a stream normed in groups, a convolution over a step's rows; retention and the gated matrix memory.
_SIGNATURES.update({
    "ti_gated_add_norm32": [_P, _P, _P, _I, _L, _P, _P, _I, _P, _P, _P, _I, _L, _P, _F, _P, _P, _I, _F, _I, _P, _I, _P, _L, _P, _P, _I, _I, _I, _P],
    "ti_conv_rows": [_P, _P, _P, _I, _P, _L, _P, _P, _I, _I, _I, _I, _P],
    "ti_retention_scan": [_P, _P, _L, _I, _I, _I, _P, _L, _P, _P, _I, _P, _F, _F, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "ti_memory_gates": [_P, _P, _P, _L, _P, _F, _P, _L, _P, _P, _I, _I, _P],
    "ti_memory_scan": [_P, _P, _P, _L, _I, _I, _I, _P, _L, _P, _F, _F, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "ti_memory_chunks": [_P, _P, _P, _P, _P, _L, _I, _I, _I, _I, _P, _L, _P, _P, _P, _I, _P, _F, _F, _P, _I, _F, _P, _P, _I, _P, _P, _I, _I, _I, _I, _I, _P],
    "ti_memory_token": [_P, _P, _P, _P, _P, _P, _L, _I, _I, _I, _I, _P, _L, _P, _P, _L, _P, _F, _P, _I, _P, _F, _F, _P, _I, _F, _P, _I, _I, _I, _I,
                        _I, _P],
})

# The update of a stream by two sublayers side by side. The state-space recurrence: inputs, one-token step, chunks of a prompt, gate and norm of its output.
_SIGNATURES.update({
    "ti_pair_add_norm32": [_P, _P, _P, _I, _L, _P, _P, _I, _L, _P, _P, _F, _F, _F, _F, _P, _P, _I, _F, _I, _I, _I, _P],
    "ti_ssm_inputs": [_P, _P, _P, _L, _I, _I, _P, _I, _P, _P, _L, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "ti_ssm_token": [_P, _P, _P, _P, _P, _L, _P, _I, _I, _I, _I, _I, _I, _I, _P],
    "ti_ssm_chunks": [_P, _P, _L, _I, _I, _I, _P, _L, _P, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "ti_ssm_chunks_tc": [_P, _P, _L, _I, _I, _I, _P, _L, _P, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _I, _P],
    "ti_ssm_gate_norm": [_P, _P, _P, _L, _P, _F, _I, _I, _I, _I, _P],
})
