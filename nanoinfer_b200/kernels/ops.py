"""Python entry points of the CUDA kernels.

Each function checks its operands (device, dtype, contiguity, sizes the kernel can take),
launches on torch's current stream and raises on any error.  Nothing here computes: a
missing CUDA library or a tensor on the CPU is an error, never a fallback.
"""
from __future__ import annotations

import ctypes
from typing import Dict, Optional

import torch

from . import build

_I, _F, _P, _LL = ctypes.c_int, ctypes.c_float, ctypes.c_void_p, ctypes.c_longlong

F32, BF16 = 0, 1
_DTYPE_CODE = {torch.float32: F32, torch.bfloat16: BF16}

_ERRORS = {-1: "bad argument", -2: "size not supported by this kernel",
           -3: "a wait inside the kernel ran out (device timeout)"}

# module -> {function: argtypes}
_SIGNATURES = {
    "elementwise": {
        "ni_embedding": [_P, _P, _I, _P, _I, _I, _I, _P],
        "ni_add_rmsnorm": [_P, _P, _I, _P, _F, _P, _I, _P, _I, _I, _P, _P, _P],
        "ni_residual_add": [_P, _P, _I, _LL, _P],
        "ni_residual_add_scaled": [_P, _P, _I, _LL, _I, _P, _P, _P],
        "ni_swiglu": [_P, _P, _I, _I, _I, _I, _P],
        "ni_swiglu_blocked": [_P, _P, _I, _I, _I, _I, _P],
    },
    "rope_kv": {
        "ni_rope_kv_write": [_P, _I, _P, _P, _P, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    },
    "attention_generic": {
        "ni_attention_generic": [_P, _I, _P, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _F, _P, _F, _I, _I, _P, _I, _P],
    },
    "gemm_f32": {
        "ni_gemm_f32": [_P, _P, _P, _I, _I, _I, _P],
        "ni_gemm_f32_heads": [_P, _I, _P, _P, _I, _I, _I, _I, _P],
    },
    "pointwise": {
        "ni_embedding_sinusoid": [_P, _P, _P, _I, _P, _P, _I, _I, _I, _P],
        "ni_cast_bf16": [_P, _P, _LL, _P],
        "ni_add_normed": [_P, _P, _I, _P, _F, _I, _I, _P, _P, _P],
        "ni_polynorm": [_P, _I, _P, _F, _P, _I, _I, _P],
        "ni_gelu_table_gate": [_P, _I, _P, _P, _I, _P, _I, _I, _I, _I, _I, _P],
        "ni_add_row": [_P, _P, _I, _I, _I, _P],
        "ni_embedding_scaled": [_P, _P, _I, _F, _P, _I, _I, _I, _P],
        "ni_scale_f32": [_P, _F, _LL, _P],
        "ni_capped_glu": [_P, _P, _I, _I, _I, _F, _F, _F, _P, _P, _P],
        "ni_concat_cast": [_P, _P, _P, _I, _I, _I, _P],
        "ni_relu_squared": [_P, _P, _I, _LL, _P],
        "ni_weighted_sum": [_P, _F, _P, _F, _P, _LL, _P],
        "ni_embedding_pairs": [_P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _I, _P, _P, _P, _P, _P, _P],
    },
    "qk_norm_rope": {
        "ni_qk_norm_rope": [_P, _I, _I, _I, _P, _P, _P, _F, _P, _P, _P, _I, _P, _F, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _F, _F, _P, _I, _P, _F, _P],
    },
    "lightning": {
        "ni_lightning_recurrence": [_P, _I, _I, _P, _LL, _P, _P, _P, _P, _I, _I, _I, _P, _LL, _I, _I, _I, _I, _P],
        "ni_linear_attention_prepare": [_P, _I, _I, _P, _P, _F, _P, _I, _I, _I, _I, _I, _P],
        "ni_retention_token_step": [_P, _I, _I, _P, _LL, _P, _P, _P, _P, _I, _I, _I, _I, _P, _P, _I, _F, _P],
        "ni_group_gated_norm": [_P, _P, _I, _I, _I, _P, _F, _P, _I, _I, _I, _I, _F, _P],
        "ni_lightning_max_chunks": [_I, _I],
        "ni_lightning_gated_norm": [_P, _P, _I, _I, _I, _P, _F, _P, _I, _I, _P],
    },
    "mlstm": {
        "ni_mlstm_token_step": [_P, _I, _P, _I, _I, _I, _P, _P, _F, _P, _LL, _P, _P, _I, _F, _P, _F, _P, _I, _I, _I, _I, _P],
        "ni_mlstm_chunk_step": [_P, _I, _I, _P, _I, _I, _I, _P, _P, _F, _P, _LL, _P, _P, _I, _I, _I, _F, _P, _F, _P, _LL, _P, _P, _P,
                                _I, _I, _I, _P],
    },
    "hyper": {
        "ni_hyper_step": [_P, _P, _I, _I, _I, _I, _I, _P, _P, _I, _P, _P, _P, _I, _I, _P, _P, _P, _P, _P, _P, _P, _P, _P],
        "ni_hyper_max_streams": [],
    },
    "difference": {
        "ni_difference_norm": [_P, _P, _I, _P, _I, _I, _I, _F, _F, _F, _P],
    },
    "conv_attention": {
        "ni_conv_qk_prepare": [_P, _I, _I, _P, _P, _P, _F, _P, _LL, _P, _P, _P, _P, _P, _I, _P, _P, _P, _P,
                               _I, _I, _I, _I, _I, _I, _I, _I, _P],
    },
    "routed": {
        "ni_route": [_P, _I, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P, _I, _I, _F, _P],
        "ni_route_layout": [_P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _P, _P, _P],
        "ni_expert_gemm": [_P, _I, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _F, _P, _P],
        "ni_expert_rows": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _F, _F, _F, _P, _P],
        "ni_route_combine": [_P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P],
        "ni_route_combine_add_normed": [_P, _P, _I, _P, _P, _P, _P, _P, _F, _I, _I, _I, _I, _I, _I, _P],
    },
    "delta_rule": {
        "ni_delta_prepare": [_P, _I, _P, _P, _P, _P, _LL, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P, _I, _P, _P, _P],
        "ni_delta_token_step": [_P, _I, _I, _I, _P, _I, _P, _I, _P, _P, _P, _P, _F, _F, _P, _LL, _P, _P, _P, _I, _I, _I, _I, _I, _I, _P, _I, _P],
        "ni_delta_token_max_dim": [],
        "ni_delta_recurrence": [_P, _P, _P, _I, _P, _LL, _P, _P, _I, _I, _I, _I, _I, _I, _P, _P],
        "ni_delta_gated_norm": [_P, _P, _I, _I, _P, _F, _F, _I, _I, _I, _I, _I, _I, _I, _P, _I, _I, _P, _I, _I, _P, _LL, _P, _P, _P],
    },
    "delta_chunk": {
        "ni_delta_chunk_recurrence": [_P, _I, _I, _P, _P, _P, _P, _I, _P, _LL, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P, _LL, _P, _P, _P],
        "ni_delta_chunk_set_wait": [_LL, _I],
        "ni_delta_chunk_max_dim": [],
    },
    "latent": {
        "ni_latent_norm_write": [_P, _I, _I, _I, _P, _F, _P, _P, _P, _P, _I, _I, _I, _I, _P],
        "ni_head_gate": [_P, _I, _P, _I, _I, _I, _I, _I, _F, _P],
        "ni_element_gate": [_P, _I, _P, _I, _I, _P, _I, _I, _I, _F, _P],
        "ni_latent_rope_write": [_P, _I, _I, _I, _P, _F, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P, _I, _P, _I, _P],
    },
    "gemv_bf16": {
        "ni_gemv_bf16": [_P, _P, _P, _I, _I, _I, _I, _P, _LL, _P, _P, _P, _I, _P, _I, _F, _P, _P, _P],
        "ni_gemv_bf16_out_tiles": [_I, _I],
        "ni_gemv_bf16_writes_handoff": [_I, _I, _I],
        "ni_gemv_bf16_reads_handoff": [_I, _I],
        "ni_gemv_norm_bf16": [_P, _P, _F, _P, _P, _P, _I, _I, _I, _I, _P, _LL, _P],
        "ni_gemv_qkv_rope": [_P, _P, _F, _P, _P, _P, _P, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P, _LL, _P, _I, _F, _P],
    },
    "gemv_ksplit": {
        "ni_gemv_ksplit": [_P, _P, _P, _I, _I, _I, _I, _P, _LL, _P, _P, _P, _I, _P, _P, _P],
        "ni_gemv_ksplit_out_tiles": [_I, _I],
        "ni_gemv_ksplit_supports": [_I, _I, _I],
    },
    "attention_decode": {
        "ni_attention_decode": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _I, _P, _P, _P, _LL, _P, _LL, _P],
        "ni_attention_decode_capped": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _F, _I, _P, _P, _P, _LL, _P, _LL, _P],
        "ni_attention_decode_masked": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _F, _I, _P, _I, _I, _P, _P, _P, _LL, _P, _LL, _P],
        "ni_attention_decode_difference": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _F, _F, _I, _I, _P, _P, _P, _LL, _P, _LL, _P],
        "ni_attention_decode_balanced": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _P, _P, _P, _LL, _P, _LL, _P],
        "ni_attention_decode_fresh_keys": [],
        "ni_attention_decode_set_cluster_merge": [_I],
        # the variant whose scratch lies in the library's own image (attention_decode_noalloc.h)
        "ni_attention_decode_noalloc": [_P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _I, _P],
    },
    "attention_prefill": {
        "ni_attention_prefill": [_P, _P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _F, _I, _P, _P],
    },
    "attention_prefill_tc": {
        "ni_attention_prefill_tc": [_P, _P, _P, _P, _I, _I, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _P, _P],
        "ni_attention_prefill_tc_masked": [_P, _P, _P, _P, _I, _I, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _I, _P, _P, _P],
        "ni_attention_prefill_tc_difference": [_P, _P, _P, _P, _I, _I, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _F, _F, _P, _P],
        "ni_attention_prefill_tc_supports": [_I, _I, _I, _I],
        "ni_attention_prefill_tc_set_wait": [_LL, _I],
    },
    "gemm_swap_tc": {
        "ni_gemm_swap_tc": [_P, _P, _P, _I, _I, _I, _I, _P, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _I, _P, _P],
        "ni_gemm_swap_tc_splits": [_I, _I, _I],
        "ni_gemm_swap_tc_scratch": [_I, _I, _I],
        "ni_gemm_swap_tc_set_wait": [_LL, _I],
    },
    "gemm_tc2": {
        "ni_gemm_tc2": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _P, _P],
        "ni_gemm_tc2_set_wait": [_LL, _I],
    },
    "gemm_tc": {
        "ni_gemm_tc": [_P, _P, _P, _I, _I, _I, _I, _P, _P],
        "ni_gemm_tc_set_wait": [_LL, _I],
    },
    "decode_fused": {
        "ni_decode_fused": [_P, _P],
        "ni_decode_fused_supports": [_I] * 9,
        "ni_decode_fused_max_rows": [],
        "ni_decode_fused_max_groups": [],
        "ni_decode_fused_blocks": [],
    },
    "sampling": {
        "ni_argmax": [_P, _P, _I, _I, _P, _P],
        "ni_repetition_penalty": [_P, _P, _P, _I, _I, _I, _P],
        "ni_sample": [_P, _P, _P, _P, _P, _P, _P, _I, _I, _P],
        "ni_sample_set_cluster": [_I],
    },
}

_libs: Dict[str, ctypes.CDLL] = {}


class KernelError(RuntimeError):
    pass


def require_cuda() -> None:
    if not torch.cuda.is_available():
        raise KernelError("nanoinfer_b200 runs on a CUDA device (sm_100a) only; "
                          "torch.cuda.is_available() is False and there is no CPU path")


def load(module: str) -> ctypes.CDLL:
    lib = _libs.get(module)
    if lib is None:
        path = build.ensure_built([module])[module]
        lib = ctypes.CDLL(path)
        for fn, argtypes in _SIGNATURES.get(module, {}).items():
            f = getattr(lib, fn)
            f.argtypes = argtypes
            f.restype = _I
        import os
        if module == "sampling" and os.environ.get("NANOINFER_B200_SAMPLE_ONE_BLOCK"):      # for comparisons
            lib.ni_sample_set_cluster(0)
        if module == "attention_decode" and os.environ.get("NANOINFER_B200_SCRATCH_MERGE"):
            lib.ni_attention_decode_set_cluster_merge(0)
        if module == "attention_decode" and lib.ni_attention_decode_fresh_keys() != DECODE_FRESH_KEYS:
            raise KernelError("attention_decode: DEC_FRESH_KEYS of the built kernel differs from ops.DECODE_FRESH_KEYS")
        if module == "delta_chunk" and lib.ni_delta_chunk_max_dim() != DELTA_CHUNK_MAX_DIM:
            raise KernelError("delta_chunk: the built kernel's largest key size differs from ops.DELTA_CHUNK_MAX_DIM")
        if module == "delta_rule" and lib.ni_delta_token_max_dim() != DELTA_TOKEN_MAX_DIM:
            raise KernelError("delta_rule: the built kernel's largest sizes differ from ops.DELTA_TOKEN_MAX_DIM")
        if module == "hyper" and lib.ni_hyper_max_streams() != HYPER_MAX_STREAMS:
            raise KernelError("hyper: HY_MAX_STREAMS of the built kernel differs from ops.HYPER_MAX_STREAMS")
        _libs[module] = lib
    return lib


def preload(modules) -> None:
    """Build (in parallel) and load the given modules ahead of their first use."""
    build.ensure_built(list(modules))
    for m in modules:
        load(m)


_sm_counts: Dict[int, int] = {}


def sm_count(device=None) -> int:
    """Streaming multiprocessors of the device (148 on a B200); every work split asks here."""
    idx = torch.cuda.current_device() if device is None else torch.device(device).index or 0
    n = _sm_counts.get(idx)
    if n is None:
        n = _sm_counts[idx] = torch.cuda.get_device_properties(idx).multi_processor_count
    return n


_launches = 0


def launch_count() -> int:
    """How many kernels of this package have been launched (or captured) so far."""
    return _launches


def _check(code: int, what: str) -> None:
    global _launches
    if code == 0:
        _launches += 1
        return
    if code < 0:
        raise KernelError(f"{what}: {_ERRORS.get(code, f'error {code}')}")
    raise KernelError(f"{what}: CUDA error {code} at launch")


def _check_plain(code: int, what: str) -> None:
    """As _check, for calls that launch nothing."""
    if code < 0:
        raise KernelError(f"{what}: {_ERRORS.get(code, f'error {code}')}")
    if code > 0:
        raise KernelError(f"{what}: CUDA error {code}")


def _stream() -> int:
    """The raw handle of torch's current stream on the current device (the C accessors: the Python
    wrapper costs more than a short kernel's launch)."""
    return torch._C._cuda_getCurrentRawStream(torch._C._cuda_getDevice())


_stream_objects: Dict[int, "torch.cuda.Stream"] = {}


def current_stream_object() -> "torch.cuda.Stream":
    """torch's current stream as an object (for Event.record), cached by raw handle."""
    raw = _stream()
    obj = _stream_objects.get(raw)
    if obj is None:
        obj = _stream_objects[raw] = torch.cuda.current_stream()
    return obj


def _dev(t: torch.Tensor, name: str, dtype=None) -> int:
    if not t.is_cuda:
        raise KernelError(f"{name} must be a CUDA tensor")
    if not t.is_contiguous():
        raise KernelError(f"{name} must be contiguous")
    if dtype is not None and t.dtype != dtype:
        raise KernelError(f"{name} must be {dtype}, found {t.dtype}")
    return t.data_ptr()


def _code(t: torch.Tensor, name: str) -> int:
    if t.dtype not in _DTYPE_CODE:
        raise KernelError(f"{name}: dtype {t.dtype} is not supported (float32 or bfloat16)")
    return _DTYPE_CODE[t.dtype]


def embedding(tokens: torch.Tensor, table: torch.Tensor, out: torch.Tensor) -> None:
    """out[t, :] = float32(table[tokens[t], :]);  tokens int32 [T], out float32 [T, d]."""
    n, d = out.shape
    if tokens.numel() != n or table.shape[1] != d:
        raise KernelError("embedding: shapes do not agree")
    _check(load("elementwise").ni_embedding(_dev(tokens, "tokens", torch.int32), _dev(table, "table"),
                                            _code(table, "table"), _dev(out, "out", torch.float32),
                                            n, d, table.shape[0], _stream()), "embedding")


class ScaledAddition:
    """An addition still pending on the residual stream whose columns have a factor and a shift of their own: the stream
    becomes h + y * scale + shift, with ``scale`` and ``shift`` float32 [d] or None.  Where a pending addition may be a
    tensor it may be one of these."""

    def __init__(self, y: torch.Tensor, scale: Optional[torch.Tensor], shift: Optional[torch.Tensor]) -> None:
        self.y, self.scale, self.shift = y, scale, shift


def _pending(delta) -> tuple:
    """(tensor, scale, shift) of a pending addition: a tensor, a ScaledAddition or None."""
    if isinstance(delta, ScaledAddition):
        d = delta.y.shape[1]
        for v in (delta.scale, delta.shift):
            if v is not None and v.numel() != d:
                raise KernelError("a pending addition's scale and shift must have its width")
        return delta.y, delta.scale, delta.shift
    return delta, None, None


def _f32_or_none(t: Optional[torch.Tensor], name: str):
    return _dev(t, name, torch.float32) if t is not None else None


def add_rmsnorm(h: torch.Tensor, delta, gain: torch.Tensor, eps: float,
                out: torch.Tensor, rows: Optional[torch.Tensor] = None) -> None:
    """Residual add fused with RMSNorm.

    h float32 [T, d]; delta [T, d], a ScaledAddition or None; gain float32 [d]; out [R, d].
    rows None: R = T, h += delta in place, out = norm(h) * gain.
    rows int32 [R]: out[r] = norm(h[rows[r]] + delta[rows[r]]) * gain, h untouched.
    """
    d = h.shape[1]
    n_out = out.shape[0]
    delta, scale, shift = _pending(delta)
    if out.shape[1] != d or gain.numel() != d:
        raise KernelError("add_rmsnorm: widths do not agree")
    if rows is None and n_out != h.shape[0]:
        raise KernelError("add_rmsnorm: out must have as many rows as h")
    if rows is not None and rows.numel() != n_out:
        raise KernelError("add_rmsnorm: rows and out do not agree")
    if delta is not None and delta.shape != h.shape:
        raise KernelError("add_rmsnorm: delta must have the shape of h")
    _check(load("elementwise").ni_add_rmsnorm(
        _dev(h, "h", torch.float32), _dev(delta, "delta") if delta is not None else None,
        _code(delta, "delta") if delta is not None else F32, _dev(gain, "gain", torch.float32),
        float(eps), _dev(out, "out"), _code(out, "out"),
        _dev(rows, "rows", torch.int32) if rows is not None else None, n_out, d, _f32_or_none(scale, "scale"),
        _f32_or_none(shift, "shift"), _stream()), "add_rmsnorm")


def residual_add(h: torch.Tensor, delta) -> None:
    """h += delta; delta [T, d] or a ScaledAddition."""
    delta, scale, shift = _pending(delta)
    if scale is not None or shift is not None:
        if delta.shape != h.shape:
            raise KernelError("residual_add: shapes do not agree")
        _check(load("elementwise").ni_residual_add_scaled(
            _dev(h, "h", torch.float32), _dev(delta, "delta"), _code(delta, "delta"), h.numel(), h.shape[1],
            _f32_or_none(scale, "scale"), _f32_or_none(shift, "shift"), _stream()), "residual_add")
        return
    if delta.shape != h.shape:
        raise KernelError("residual_add: shapes do not agree")
    _check(load("elementwise").ni_residual_add(_dev(h, "h", torch.float32), _dev(delta, "delta"),
                                               _code(delta, "delta"), h.numel(), _stream()),
           "residual_add")


def swiglu(gate_up: torch.Tensor, out: torch.Tensor, blocked: bool = False, gelu: bool = False) -> None:
    """out[t, i] = silu(gate[t, i]) * up[t, i] (``gelu``: the tanh form of gelu instead of silu).  Plain layout: gate_up = [gate | up] along the
    columns.  Blocked layout (I a multiple of 8): columns in blocks of 8 gate values followed by
    their 8 up values."""
    n, inter = out.shape
    if gate_up.shape != (n, 2 * inter) or gate_up.dtype != out.dtype:
        raise KernelError("swiglu: gate_up must be [T, 2I] of out's dtype")
    if blocked and inter % 8:
        raise KernelError("swiglu: the blocked layout needs I to be a multiple of 8")
    fn = load("elementwise").ni_swiglu_blocked if blocked else load("elementwise").ni_swiglu
    _check(fn(_dev(gate_up, "gate_up"), _dev(out, "out"), _code(out, "out"), n, inter, 1 if gelu else 0, _stream()), "swiglu")


def rope_kv_write(qkv: torch.Tensor, q_out: torch.Tensor, k_pages: Optional[torch.Tensor],
                  v_pages: Optional[torch.Tensor], positions: torch.Tensor,
                  seq_of_token: torch.Tensor, block_table: torch.Tensor, inv_freq: torch.Tensor,
                  n_q_heads: int, n_kv_heads: int, head_dim: int, rotary_dim: int,
                  interleaved: bool, page_size: int) -> None:
    """Rotate q and k of the fused projection qkv [T, (Hq + 2 Hkv) hd]; q -> q_out
    [T, Hq hd]; k (rotated) and v -> pages [P, Hkv, page_size, hd] unless k_pages is None."""
    n = qkv.shape[0]
    write = k_pages is not None
    if qkv.shape[1] != (n_q_heads + 2 * n_kv_heads) * head_dim or q_out.shape != (n, n_q_heads * head_dim):
        raise KernelError("rope_kv_write: widths do not agree with the head counts")
    if q_out.dtype != qkv.dtype or (write and (k_pages.dtype != qkv.dtype or v_pages.dtype != qkv.dtype)):
        raise KernelError("rope_kv_write: all operands must share one dtype")
    if write and tuple(k_pages.shape[1:]) != (n_kv_heads, page_size, head_dim):
        raise KernelError("rope_kv_write: pages must be [P, Hkv, page_size, head_dim]")
    if inv_freq.numel() != rotary_dim // 2 and rotary_dim > 0:
        raise KernelError("rope_kv_write: inv_freq must have rotary_dim / 2 entries")
    _check(load("rope_kv").ni_rope_kv_write(
        _dev(qkv, "qkv"), _code(qkv, "qkv"), _dev(q_out, "q_out"),
        _dev(k_pages, "k_pages") if write else None, _dev(v_pages, "v_pages") if write else None,
        _dev(positions, "positions", torch.int32), _dev(seq_of_token, "seq_of_token", torch.int32),
        _dev(block_table, "block_table", torch.int32), block_table.shape[1],
        _dev(inv_freq, "inv_freq", torch.float32), n, n_q_heads, n_kv_heads, head_dim, rotary_dim,
        1 if interleaved else 0, page_size, 1 if write else 0, _stream()), "rope_kv_write")


def _sinks(sink, n_q_heads: int, device):
    """The sinks of an attention call as float32 [Hq] on the device, or None: ``sink`` is None or False (none), True (a
    key of score 0 for every head, so that one is added to the denominators) or that tensor."""
    if sink is None or sink is False:
        return None
    if sink is True:
        return torch.zeros(n_q_heads, dtype=torch.float32, device=device)
    if sink.numel() != n_q_heads:
        raise KernelError("attention: one sink per query head")
    return sink


def attention_generic(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
                      out: torch.Tensor, positions: torch.Tensor, seq_of_token: torch.Tensor,
                      block_table: torch.Tensor, n_q_heads: int, n_kv_heads: int, head_dim: int,
                      page_size: int, window: Optional[int], scale: float,
                      token_list: Optional[torch.Tensor] = None, head_slopes: Optional[torch.Tensor] = None,
                      score_cap: float = 0.0, value_dim: Optional[int] = None, chunk: int = 0,
                      sink=None, maps: int = 1) -> None:
    """The plain attention kernel (any dtype, any head size up to 1,024).  ``token_list``
    int32 [n] restricts it to those tokens of the step.  ``head_slopes`` float32 [Hq] adds
    slope[h] * (key position - query position) to the scaled scores of head h.  ``score_cap`` c > 0
    bounds the scaled scores: s <- c * tanh(s / c).  ``value_dim``: the size of a value where it differs
    from the keys' (value pages [P, Hkv, page_size, value_dim], out [T, Hq * value_dim]).  ``chunk`` c > 0: a token at
    position p sees only the keys from p - p % c on.  ``sink`` float32 [Hq] (or True for zeros): exp(sink[h]) is added to
    the softmax's denominator of head h.  ``maps`` = m > 1: every head has m attention maps over the same values; ``n_q_heads`` counts maps (head h's map i is row h m + i of
    q), and a key row holds m parts of ``head_dim`` side by side.  ``out`` may be float32 where the rest is bfloat16."""
    if head_slopes is not None and head_slopes.numel() != n_q_heads:
        raise KernelError("attention: one slope per query head")
    n = q.shape[0]
    v_dim = head_dim if value_dim is None else int(value_dim)
    if q.shape != (n, n_q_heads * head_dim) or out.shape != (n, n_q_heads * v_dim):
        raise KernelError("attention: q must be [T, Hq * head_dim] and out [T, Hq * value_dim]")
    if not (q.dtype == k_pages.dtype == v_pages.dtype) or out.dtype not in (q.dtype, torch.float32):
        raise KernelError("attention: all operands must share one dtype (the output may be float32)")
    if head_dim > 1024 or v_dim > 1024 or v_dim <= 0:
        raise KernelError(f"attention: head_dim {head_dim} or value_dim {v_dim} beyond 1,024 is not supported")
    if k_pages.shape[-1] != maps * head_dim or v_pages.shape[-1] != v_dim:
        raise KernelError("attention: the pages' rows must have the keys' and the values' sizes")
    sink = _sinks(sink, n_q_heads, q.device)
    _check(load("attention_generic").ni_attention_generic(
        _dev(q, "q"), _code(q, "q"), _dev(k_pages, "k_pages"), _dev(v_pages, "v_pages"),
        _dev(out, "out"), _code(out, "out"), _dev(token_list, "token_list", torch.int32) if token_list is not None else None,
        _dev(positions, "positions", torch.int32),
        _dev(seq_of_token, "seq_of_token", torch.int32), _dev(block_table, "block_table", torch.int32),
        block_table.shape[1], n if token_list is None else token_list.numel(), n_q_heads, n_kv_heads, head_dim, page_size,
        int(window) if window else 0, float(scale),
        _dev(head_slopes, "head_slopes", torch.float32) if head_slopes is not None else None, float(score_cap),
        v_dim, int(chunk or 0), _f32_or_none(sink, "sink"), int(maps), _stream()), "attention_generic")


def gemm_f32(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """out[M, N] = x[M, K] . w[N, K]^T, all float32, plain FP32 arithmetic."""
    m, k = x.shape
    n = w.shape[0]
    if w.shape[1] != k or out.shape != (m, n):
        raise KernelError("gemm_f32: shapes do not agree")
    _check(load("gemm_f32").ni_gemm_f32(_dev(x, "x", torch.float32), _dev(w, "w", torch.float32),
                                        _dev(out, "out", torch.float32), m, n, k, _stream()), "gemm_f32")


def gemm_f32_heads(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """One product per head, plain FP32: out[m, h, :] = x[m, h, :] . w[h]^T with x [M, H K] (its rows may
    be some columns of a wider matrix), w [H, N, K], out [M, H N], all float32."""
    h, n, k = w.shape
    m = x.shape[0]
    if x.shape != (m, h * k) or out.shape != (m, h * n):
        raise KernelError("gemm_f32_heads: shapes do not agree")
    if not x.is_cuda or x.dtype != torch.float32 or x.stride(1) != 1 or x.stride(0) < h * k:
        raise KernelError("gemm_f32_heads: x must be float32 rows on the device, each row contiguous")
    _check(load("gemm_f32").ni_gemm_f32_heads(x.data_ptr(), x.stride(0), _dev(w, "w", torch.float32),
                                              _dev(out, "out", torch.float32), m, n, k, h, _stream()), "gemm_f32_heads")


def embedding_sinusoid(tokens: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, inv_freq: torch.Tensor,
                       out: torch.Tensor) -> None:
    """out[t, 2i] = table[tokens[t], 2i] + sin(p f_i), out[t, 2i+1] = table[tokens[t], 2i+1] + cos(p f_i) with
    p = positions[t], f = inv_freq float32 [ceil(d / 2)]; out float32 [T, d]."""
    n, d = out.shape
    if tokens.numel() != n or positions.numel() != n or table.shape[1] != d or inv_freq.numel() != (d + 1) // 2:
        raise KernelError("embedding_sinusoid: shapes do not agree")
    _check(load("pointwise").ni_embedding_sinusoid(
        _dev(tokens, "tokens", torch.int32), _dev(positions, "positions", torch.int32), _dev(table, "table"),
        _code(table, "table"), _dev(inv_freq, "inv_freq", torch.float32), _dev(out, "out", torch.float32), n, d,
        table.shape[0], _stream()), "embedding_sinusoid")


def cast_bf16(x: torch.Tensor, out: torch.Tensor) -> None:
    """out = bfloat16(x) for float32 x of the same shape."""
    if x.shape != out.shape:
        raise KernelError("cast_bf16: shapes do not agree")
    _check(load("pointwise").ni_cast_bf16(_dev(x, "x", torch.float32), _dev(out, "out", torch.bfloat16), x.numel(),
                                          _stream()), "cast_bf16")


def add_normed(h: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float, bias: Optional[torch.Tensor] = None,
               rounded: Optional[torch.Tensor] = None) -> None:
    """h += z / sqrt(mean(z^2) + eps) * weight, row by row, with z = y (+ ``bias`` float32 [d], if given); h float32
    [T, d], weight float32 [d].  ``rounded`` (bfloat16 [T, d]): also receives the updated h, rounded."""
    n, d = h.shape
    if y.shape != h.shape or weight.numel() != d or (bias is not None and bias.numel() != d) or \
            (rounded is not None and rounded.shape != h.shape):
        raise KernelError("add_normed: shapes do not agree")
    _check(load("pointwise").ni_add_normed(_dev(h, "h", torch.float32), _dev(y, "y"), _code(y, "y"),
                                           _dev(weight, "weight", torch.float32), float(eps), n, d,
                                           _dev(bias, "bias", torch.float32) if bias is not None else None,
                                           _dev(rounded, "rounded", torch.bfloat16) if rounded is not None else None,
                                           _stream()), "add_normed")


def polynorm(z: torch.Tensor, coef: torch.Tensor, eps: float, out: torch.Tensor) -> None:
    """out = c1 R(z) + c2 R(z * z) + c3 R(z * z * z) + c0 per row, where R divides a row by its root mean square
    (eps under the root); coef = (c1, c2, c3, c0)
    float32 on the device; z and out [T, n] of one dtype."""
    if z.shape != out.shape or z.dtype != out.dtype or coef.numel() != 4:
        raise KernelError("polynorm: shapes or dtypes do not agree")
    _check(load("pointwise").ni_polynorm(_dev(z, "z"), _code(z, "z"), _dev(coef, "coef", torch.float32), float(eps),
                                         _dev(out, "out"), z.shape[0], z.shape[1], _stream()), "polynorm")


def gelu_table_gate(gate: torch.Tensor, tokens: torch.Tensor, table: torch.Tensor, first: int, out: torch.Tensor) -> None:
    """out[t, j] = gelu_tanh(gate[t, j]) * table[tokens[t], first + j]; gate, out [T, n]; table [vocab, stride]."""
    n_rows, n = gate.shape
    if out.shape != gate.shape or out.dtype != gate.dtype or table.dtype != gate.dtype or tokens.numel() != n_rows:
        raise KernelError("gelu_table_gate: shapes or dtypes do not agree")
    _check(load("pointwise").ni_gelu_table_gate(
        _dev(gate, "gate"), _code(gate, "gate"), _dev(tokens, "tokens", torch.int32), _dev(table, "table"),
        _code(table, "table"), _dev(out, "out"), n_rows, n, int(first), table.shape[1], table.shape[0], _stream()),
        "gelu_table_gate")


def delta_prepare(proj, conv_w, a_log, dt_bias, state, seq_of_token, cu_q, slots, n_seqs, n_q_heads_kv, n_heads, dim,
                  vdim, taps, qkv, gates, col0: int = 0, b_col: Optional[int] = None, z=None) -> None:
    """The gated delta rule's per-token inputs from the fused projection ``proj`` ([T, ld], float32 or bfloat16; from column
    ``col0`` on q | k | v; b at ``b_col``): convolution + silu, unit q and k -> qkv [T, C]; decay and beta -> gates
    [T, H, 2].  Without ``z`` the decays are one per head, their logits at the columns after b, and ``b_col`` defaults to
    the column after q | k | v and a gate of H V.  ``z`` (float32 [T, *], the first H D columns): the decays are one per
    head and key channel; z holds their logits and, afterwards, the decays; ``dt_bias`` then has H D entries.
    It reads each request's convolution history in ``state`` (float32 [slots, H D V + (taps - 1) C]); the new
    history is written by delta_gated_norm, which must follow in the same step."""
    n = proj.shape[0]
    c = 2 * n_q_heads_kv * dim + n_heads * vdim
    if b_col is None:
        b_col = col0 + c + n_heads * vdim
    a_rel = b_col - col0 + n_heads if z is None else -1
    if qkv.shape != (n, c) or gates.shape != (n, n_heads, 2) or conv_w.shape != (c, taps):
        raise KernelError("delta_prepare: shapes do not agree")
    if proj.shape[1] < max(col0 + c, b_col + n_heads * (2 if z is None else 1)):
        raise KernelError("delta_prepare: the projection has too few columns")
    if dt_bias.numel() != n_heads * (dim if z is not None else 1) or a_log.numel() != n_heads or \
            (z is not None and (z.shape[0] != n or z.shape[1] < n_heads * dim)):
        raise KernelError("delta_prepare: the decay's constants or logits have another size")
    if state.shape[1] != n_heads * dim * vdim + (taps - 1) * c:
        raise KernelError("delta_prepare: the state has another size")
    f32 = torch.float32
    _check(load("delta_rule").ni_delta_prepare(
        _dev(proj, "proj") + col0 * proj.element_size(), _code(proj, "proj"), _dev(conv_w, "conv_w", f32),
        _dev(a_log, "a_log", f32), _dev(dt_bias, "dt_bias", f32),
        _dev(state, "state", f32), state.shape[1], _dev(seq_of_token, "seq_of_token", torch.int32),
        _dev(cu_q, "cu_q", torch.int32), _dev(slots, "slots", torch.int32), n, n_seqs, n_q_heads_kv, n_heads, dim, vdim,
        taps, proj.shape[1], b_col - col0, a_rel, _f32_or_none(z, "z"), z.shape[1] if z is not None else 0,
        _dev(qkv, "qkv", f32), _dev(gates, "gates", f32), _stream()), "delta_prepare")


def delta_recurrence(qkv, gates, state, cu_q, slots, n_seqs, n_q_heads_kv, n_heads, dim, vdim, out, z=None) -> None:
    """Per head and token, in order: the state M [D, V] decays (M *= decay), the error e = beta * (v - k M) is
    written back (M += outer(k, e)) and the token reads y = q M - for every token of every request;
    S float32 [H, D, V] at the start of each row of ``state``; out float32 [T, H V].  ``z``: decays per head and key channel,
    as delta_prepare leaves them (they multiply the rows of M)."""
    f32 = torch.float32
    if out.shape != (qkv.shape[0], n_heads * vdim) or (z is not None and (z.shape[0] != out.shape[0] or z.shape[1] < n_heads * dim)):
        raise KernelError("delta_recurrence: out must be [T, H V] (and z [T, H D] or wider)")
    _check(load("delta_rule").ni_delta_recurrence(
        _dev(qkv, "qkv", f32), _dev(gates, "gates", f32), _f32_or_none(z, "z"), z.shape[1] if z is not None else 0,
        _dev(state, "state", f32), state.shape[1], _dev(cu_q, "cu_q", torch.int32), _dev(slots, "slots", torch.int32),
        qkv.shape[0], n_seqs, n_q_heads_kv, n_heads, dim, vdim, _dev(out, "out", f32), _stream()), "delta_recurrence")


def delta_gated_norm(o, proj, weight, eps, n_q_heads_kv, n_heads, dim, vdim, y, state, cu_q, slots, n_seqs, taps, col0: int = 0,
                     gate=None, gate_col: Optional[int] = None, sigmoid: bool = False, scale: float = 1.0, y_col: int = 0) -> None:
    """y[t, y_col + h vdim ..] = o[t, h, :] / rms * weight * silu(gate[t, h, :]) * scale (``sigmoid``: instead of silu); gate
    = columns ``gate_col`` on of the float32 tensor ``gate`` (default: of proj, behind q | k | v); and each request's new
    convolution history (its last taps - 1 rows of ``proj``, columns ``col0`` on) into ``state``."""
    n = o.shape[0]
    f32 = torch.float32
    hv, c = n_heads * vdim, 2 * n_q_heads_kv * dim + n_heads * vdim
    gate = proj if gate is None else gate
    gate_col = col0 + c if gate_col is None else gate_col
    if o.shape != (n, hv) or y.shape[0] != n or y.shape[1] < y_col + hv or weight.numel() != vdim or gate.shape[0] != n or \
            gate.shape[1] < gate_col + hv or proj.shape[0] != n or proj.shape[1] < col0 + c:
        raise KernelError("delta_gated_norm: shapes do not agree")
    _check(load("delta_rule").ni_delta_gated_norm(
        _dev(o, "o", f32), _dev(gate, "gate", f32) + gate_col * 4, gate.shape[1], 1 if sigmoid else 0,
        _dev(weight, "weight", f32), float(eps), float(scale), n, n_seqs, n_q_heads_kv, n_heads, dim, vdim, taps,
        _dev(y, "y") + y_col * y.element_size(), _code(y, "y"), y.shape[1], _dev(proj, "proj") + col0 * proj.element_size(),
        _code(proj, "proj"), proj.shape[1], _dev(state, "state", f32), state.shape[1], _dev(cu_q, "cu_q", torch.int32),
        _dev(slots, "slots", torch.int32), _stream()), "delta_gated_norm")


DELTA_CHUNK_MAX_DIM = 128      # the largest key size that the chunked delta rule takes


def delta_chunk_buffer_bytes(n_tokens: int, n_seqs: int, n_heads: int, dim: int, vdim: int) -> int:
    """Bytes of the buffer that delta_chunk_recurrence needs for a step."""
    f = load("delta_chunk").ni_delta_chunk_buffer_bytes
    f.restype, f.argtypes = ctypes.c_longlong, [_I] * 5
    return int(f(n_tokens, n_seqs, n_heads, dim, vdim))


def delta_chunk_recurrence(proj, col0, b_col, conv_w, a_log, dt_bias, z, state, cu_q, slots, n_seqs, max_q_len, n_q_heads_kv, n_heads,
                           dim, vdim, taps, buf, out) -> None:
    """What delta_prepare and delta_recurrence do with decays per key channel, for prompt portions of a bfloat16 projection
    (``proj`` [T, *], q | k | v from column ``col0`` on, beta's logits at ``b_col``; ``z`` float32 [T, *]: the decays' logits
    in its first H D columns, left as they are): chunks of 32 tokens, their products on the tensor cores with every FP32
    operand split into two bfloat16 halves.  ``max_q_len``: the most tokens that one request brings; ``buf``:
    delta_chunk_buffer_bytes bytes on the device.  delta_gated_norm must follow (it moves the convolution history on)."""
    f32 = torch.float32
    n = proj.shape[0]
    c = 2 * n_q_heads_kv * dim + n_heads * vdim
    if out.shape != (n, n_heads * vdim) or z.shape[0] != n or z.shape[1] < n_heads * dim or b_col < col0 or \
            proj.shape[1] < max(col0 + c, b_col + n_heads) or conv_w.shape != (c, taps) or a_log.numel() != n_heads or \
            dt_bias.numel() != n_heads * dim or state.shape[1] != n_heads * dim * vdim + (taps - 1) * c:
        raise KernelError("delta_chunk_recurrence: shapes do not agree")
    _check(load("delta_chunk").ni_delta_chunk_recurrence(
        _dev(proj, "proj", torch.bfloat16) + 2 * col0, proj.shape[1], b_col - col0, _dev(conv_w, "conv_w", f32),
        _dev(a_log, "a_log", f32), _dev(dt_bias, "dt_bias", f32), _dev(z, "z", f32), z.shape[1], _dev(state, "state", f32),
        state.shape[1], _dev(cu_q, "cu_q", torch.int32), _dev(slots, "slots", torch.int32), n, n_seqs, int(max_q_len), n_q_heads_kv,
        n_heads, dim, vdim, taps, _dev(buf, "buf"), buf.numel() * buf.element_size(), _dev(out, "out", f32),
        _error_word(proj.device).data_ptr(), _stream()), "delta_chunk_recurrence")


DELTA_TOKEN_MAX_DIM = 128      # the largest key and value sizes whose state a block of the token kernel holds in registers


def delta_token_step(proj, col0, b_col, thin_col, w_decay, w_gate, conv_w, a_log, dt_bias, norm_w, eps, scale, state, cu_q, slots,
                     tickets, n_seqs, n_q_heads_kv, n_heads, dim, vdim, taps, y, y_col: int = 0) -> None:
    """A step of single tokens of the delta rule with decays per key channel in one launch: from ``proj`` (float32 [T, *], from
    column ``col0`` on q | k | v, beta's logits at ``b_col``, the thin first products of decay and gate at ``thin_col``) to
    the gated, normed read-outs in columns ``y_col`` on of ``y`` (bfloat16); the thin second products with ``w_decay``
    (bfloat16 [H D, ra]) and ``w_gate`` ([H V, rg]; ra and rg multiples of 8) inside.  The state moves on, convolution
    history included.  tickets: int32 zeros, at least n_seqs * q/k heads (left zero)."""
    n = proj.shape[0]
    f32, bf, i32 = torch.float32, torch.bfloat16, torch.int32
    c, hd, hv = 2 * n_q_heads_kv * dim + n_heads * vdim, n_heads * dim, n_heads * vdim
    ra, rg = w_decay.shape[1], w_gate.shape[1]
    if n != n_seqs or y.shape[0] != n or y.shape[1] < y_col + hv or w_decay.shape[0] != hd or w_gate.shape[0] != hv or \
            conv_w.shape != (c, taps) or a_log.numel() != n_heads or dt_bias.numel() != hd or norm_w.numel() != vdim or \
            proj.shape[1] < max(col0 + c, b_col + n_heads, thin_col + ra + rg) or min(b_col, thin_col) < col0:
        raise KernelError("delta_token_step: shapes do not agree")
    if state.shape[1] != hd * vdim + (taps - 1) * c or tickets.numel() < n_seqs * n_q_heads_kv:
        raise KernelError("delta_token_step: the state has another size, or too few tickets")
    _check(load("delta_rule").ni_delta_token_step(
        _dev(proj, "proj", f32) + 4 * col0, proj.shape[1], b_col - col0, thin_col - col0, _dev(w_decay, "w_decay", bf), ra,
        _dev(w_gate, "w_gate", bf), rg, _dev(conv_w, "conv_w", f32), _dev(a_log, "a_log", f32), _dev(dt_bias, "dt_bias", f32),
        _dev(norm_w, "norm_w", f32), float(eps), float(scale), _dev(state, "state", f32), state.shape[1], _dev(cu_q, "cu_q", i32),
        _dev(slots, "slots", i32), _dev(tickets, "tickets", i32), n_seqs, n_q_heads_kv, n_heads, dim, vdim, taps,
        _dev(y, "y", bf) + 2 * y_col, y.shape[1], _stream()), "delta_token_step")


def latent_norm_write(proj, col0, rank, weight, eps, pages, positions, seq_of_token, block_table, page_size) -> None:
    """pages[page of t, place of t, :] = RMSNorm(proj[t, col0 : col0 + rank]) * weight; pages [P, page_size, rank]."""
    n = proj.shape[0]
    if tuple(pages.shape[1:]) != (page_size, rank) or pages.dtype != proj.dtype or weight.numel() != rank:
        raise KernelError("latent_norm_write: pages must be [P, page_size, rank] of proj's dtype")
    _check(load("latent").ni_latent_norm_write(
        _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], int(col0), _dev(weight, "weight", torch.float32),
        float(eps), _dev(pages, "pages"), _dev(positions, "positions", torch.int32),
        _dev(seq_of_token, "seq_of_token", torch.int32), _dev(block_table, "block_table", torch.int32),
        block_table.shape[1], n, rank, page_size, _stream()), "latent_norm_write")


def latent_rope_write(proj, col0, rank, rot_dim, weight, eps, pages, positions, seq_of_token, block_table, page_size,
                      inv_freq, interleaved, q, n_heads) -> None:
    """A latent cache row with a rotated key part: pages[page of t, place of t, :] = [RMSNorm(proj[t, col0 : col0 +
    rank]) * weight | rot(proj[t, col0 + rank : col0 + rank + rot_dim])], pages [P, page_size, rank + rot_dim] (None:
    nothing is written); the last rot_dim dimensions of every head of q [T, H (rank + rot_dim)] are rotated in place.
    Pairs (2i, 2i + 1) if ``interleaved`` else (i, i + rot_dim / 2); angle float(position) * inv_freq[i]."""
    n = proj.shape[0]
    w = rank + rot_dim
    if (pages is not None and (tuple(pages.shape[1:]) != (page_size, w) or pages.dtype != proj.dtype)) or \
            weight.numel() != rank or tuple(q.shape) != (n, n_heads * w) or q.dtype != proj.dtype or \
            (rot_dim > 0 and inv_freq.numel() != rot_dim // 2):
        raise KernelError("latent_rope_write: pages must be [P, page_size, rank + rot_dim] and q [T, H (rank + rot_dim)] of proj's dtype")
    _check(load("latent").ni_latent_rope_write(
        _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], int(col0), _dev(weight, "weight", torch.float32),
        float(eps), _dev(pages, "pages") if pages is not None else None, _dev(positions, "positions", torch.int32),
        _dev(seq_of_token, "seq_of_token", torch.int32), _dev(block_table, "block_table", torch.int32),
        block_table.shape[1], n, rank, rot_dim, page_size, _dev(inv_freq, "inv_freq", torch.float32),
        1 if interleaved else 0, _dev(q, "q"), n_heads, _stream()), "latent_rope_write")


def head_gate(x, proj, col0, n_heads, vdim, scale: float = 1.0) -> None:
    """x[t, h, :] *= sigmoid(proj[t, col0 + h]) * scale in place; x [T, H V]."""
    n = x.shape[0]
    if x.shape[1] != n_heads * vdim or proj.shape[0] != n or proj.dtype != x.dtype:
        raise KernelError("head_gate: shapes or dtypes do not agree")
    _check(load("latent").ni_head_gate(_dev(x, "x"), _code(x, "x"), _dev(proj, "proj"), proj.shape[1], int(col0), n,
                                       n_heads, vdim, float(scale), _stream()), "head_gate")


def element_gate(x, gate, col0, out=None, out_col: int = 0, scale: float = 1.0) -> None:
    """out[t, out_col + i] = x[t, i] * sigmoid(gate[t, col0 + i]) * scale for every column i of x [T, n]; ``gate`` [T, *] of
    x's dtype or float32; ``out`` (default x itself) [T, *] of x's dtype."""
    n_rows, n = x.shape
    out = x if out is None else out
    if gate.shape[0] != n_rows or gate.shape[1] < col0 + n or out.shape[0] != n_rows or out.shape[1] < out_col + n or \
            out.dtype != x.dtype or gate.dtype not in (x.dtype, torch.float32):
        raise KernelError("element_gate: shapes or dtypes do not agree")
    _check(load("latent").ni_element_gate(
        _dev(x, "x"), _code(x, "x"), _dev(gate, "gate") + col0 * gate.element_size(), _code(gate, "gate"), gate.shape[1],
        _dev(out, "out") + out_col * out.element_size(), out.shape[1], n_rows, n, float(scale), _stream()), "element_gate")


def embedding_scaled(tokens: torch.Tensor, table: torch.Tensor, scale: float, out: torch.Tensor) -> None:
    """out[t, :] = float32(table[tokens[t], :]) * scale;  tokens int32 [T], out float32 [T, d]."""
    n, d = out.shape
    if tokens.numel() != n or table.shape[1] != d:
        raise KernelError("embedding_scaled: shapes do not agree")
    _check(load("pointwise").ni_embedding_scaled(_dev(tokens, "tokens", torch.int32), _dev(table, "table"),
                                                 _code(table, "table"), float(scale), _dev(out, "out", torch.float32),
                                                 n, d, table.shape[0], _stream()), "embedding_scaled")


def embedding_pairs(tokens, table, pairs, out, buckets, mul_prev, mul_cur, positions, seq_of_token, cu_q, slots, last) -> None:
    """out[t, :] = float32(table[tokens[t]]) + float32(pairs[r]) with r = (previous token * mul_prev + token * mul_cur) mod
    buckets, or r = buckets for a token at position 0; the token before a step's first one is read from ``last``
    (int32 [slots], one per request slot), which is then set to the request's last token of this step."""
    n, d = out.shape
    if tokens.numel() != n or table.shape[1] != d or tuple(pairs.shape) != (buckets + 1, d) or pairs.dtype != table.dtype:
        raise KernelError("embedding_pairs: shapes or dtypes do not agree")
    i32 = torch.int32
    _check(load("pointwise").ni_embedding_pairs(
        _dev(tokens, "tokens", i32), _dev(table, "table"), _dev(pairs, "pairs"), _code(table, "table"),
        _dev(out, "out", torch.float32), n, d, table.shape[0], int(buckets), int(mul_prev), int(mul_cur),
        _dev(positions, "positions", i32), _dev(seq_of_token, "seq_of_token", i32), _dev(cu_q, "cu_q", i32),
        _dev(slots, "slots", i32), _dev(last, "last", i32), _stream()), "embedding_pairs")


def weighted_sum(a: torch.Tensor, sa: float, b: torch.Tensor, sb: float, out: torch.Tensor) -> None:
    """out = sa * a + sb * b, element by element; all float32 of one shape (out may be a or b)."""
    if a.shape != b.shape or out.shape != a.shape:
        raise KernelError("weighted_sum: shapes do not agree")
    f32 = torch.float32
    _check(load("pointwise").ni_weighted_sum(_dev(a, "a", f32), float(sa), _dev(b, "b", f32), float(sb), _dev(out, "out", f32),
                                             a.numel(), _stream()), "weighted_sum")


def add_row(h: torch.Tensor, row: torch.Tensor) -> None:
    """h[t, :] += row for every t; h float32 [T, d], row [d] (float32 or bfloat16)."""
    n, d = h.shape
    if row.numel() != d:
        raise KernelError("add_row: the row must have the width of h")
    _check(load("pointwise").ni_add_row(_dev(h, "h", torch.float32), _dev(row, "row"), _code(row, "row"), n, d, _stream()),
           "add_row")


def scale_f32(x: torch.Tensor, factor: float) -> None:
    """x *= factor in place; x float32."""
    _check(load("pointwise").ni_scale_f32(_dev(x, "x", torch.float32), float(factor), x.numel(), _stream()), "scale_f32")


def capped_glu(gate_up: torch.Tensor, out: torch.Tensor, limit: float, slope: float, shift: float,
               row_scale: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None) -> None:
    """out = g * sigmoid(slope * g) * (u + shift) with g = min(r gate + b_gate, limit), u = clamp(r up + b_up, -limit,
    limit); gate_up = [gate | up] [T, 2I], out [T, I], one dtype; ``row_scale`` float32 [T]: r per row (else 1) - what
    the unit computes when its input was multiplied by r; ``bias`` float32 [2I] (gate then up; else none)."""
    n, inter = out.shape
    if gate_up.shape != (n, 2 * inter) or gate_up.dtype != out.dtype or (row_scale is not None and row_scale.numel() != n) \
            or (bias is not None and bias.numel() != 2 * inter):
        raise KernelError("capped_glu: gate_up must be [T, 2I] of out's dtype (row_scale [T], bias [2I])")
    _check(load("pointwise").ni_capped_glu(_dev(gate_up, "gate_up"), _dev(out, "out"), _code(out, "out"), n, inter,
                                           float(limit), float(slope), float(shift),
                                           _dev(row_scale, "row_scale", torch.float32) if row_scale is not None else None,
                                           _dev(bias, "bias", torch.float32) if bias is not None else None,
                                           _stream()), "capped_glu")


def concat_cast(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor) -> None:
    """out[t] = [a[t] | b[t]] in out's dtype; a, b float32 [T, d], out [T, 2d]."""
    n, d = a.shape
    if b.shape != a.shape or out.shape != (n, 2 * d):
        raise KernelError("concat_cast: shapes do not agree")
    _check(load("pointwise").ni_concat_cast(_dev(a, "a", torch.float32), _dev(b, "b", torch.float32), _dev(out, "out"),
                                            _code(out, "out"), n, d, _stream()), "concat_cast")


def relu_squared(z: torch.Tensor, out: torch.Tensor) -> None:
    """out = max(z, 0)^2 element by element; one dtype."""
    if z.shape != out.shape or z.dtype != out.dtype:
        raise KernelError("relu_squared: shapes or dtypes do not agree")
    _check(load("pointwise").ni_relu_squared(_dev(z, "z"), _dev(out, "out"), _code(out, "out"), z.numel(), _stream()),
           "relu_squared")


def qk_norm_rope(qkv, bias, q_gain, k_gain, eps, positions, seq_of_token, block_table, inv_freq, magnitude, q_out,
                 k_pages, v_pages, n_heads, n_kv_heads, head_dim, value_dim, rotary_dim, page_size, head_unit=False,
                 col0=0, temperature=None, first_values=None) -> None:
    """From the fused projection ``qkv`` [T, ld] (columns q | k | v): + ``bias`` (float32 over those columns, or
    None); RMS norm of all the row's query values together and of all its key values together (``q_gain`` float32
    [H hd], ``k_gain`` float32 [Hkv hd]; both None: no norm); rotation of the first ``rotary_dim`` dimensions of every
    head, dimension i paired with i + rotary_dim / 2, cosine and sine times ``magnitude``; with ``head_unit`` every
    head of q and k is then divided by its own root mean square (``eps`` inside the root, no weight); queries -> q_out [T, H hd],
    keys -> k_pages [P, Hkv, page_size, hd], values -> v_pages [P, Hkv, page_size, value_dim] (None: nothing written).
    The columns start at ``col0`` of qkv, which may be float32 where q_out and the pages are bfloat16.  ``temperature``
    (coef, every): the finished query times 1 + coef ln(1 + floor((position + 1) / every)).  ``first_values`` (rows, column,
    bias, lambda): v <- (1 - lambda) v + lambda (rows[t, column : column + Hkv value_dim] + bias), rows [T, *] of qkv's
    dtype, bias float32 [Hkv value_dim] or None."""
    n = qkv.shape[0]
    f32, i32 = torch.float32, torch.int32
    cols = (n_heads + n_kv_heads) * head_dim + n_kv_heads * value_dim
    write = k_pages is not None
    if qkv.shape[1] < col0 + cols or q_out.shape != (n, n_heads * head_dim) or (q_out.dtype != qkv.dtype and qkv.dtype != f32):
        raise KernelError("qk_norm_rope: shapes or dtypes do not agree")
    if write and (tuple(k_pages.shape[1:]) != (n_kv_heads, page_size, head_dim) or k_pages.dtype != q_out.dtype
                  or tuple(v_pages.shape[1:]) != (n_kv_heads, page_size, value_dim) or v_pages.dtype != q_out.dtype):
        raise KernelError("qk_norm_rope: pages must be [P, Hkv, page_size, head_dim] and [P, Hkv, page_size, value_dim]")
    if (bias is not None and bias.numel() != cols) or (q_gain is None) != (k_gain is None) or \
            (q_gain is not None and (q_gain.numel() != n_heads * head_dim or k_gain.numel() != n_kv_heads * head_dim)):
        raise KernelError("qk_norm_rope: the bias or a gain has another size")
    if rotary_dim > 0 and inv_freq.numel() != rotary_dim // 2:
        raise KernelError("qk_norm_rope: inv_freq must have rotary_dim / 2 entries")
    coef, every = temperature if temperature is not None else (0.0, 1.0)
    first, first_ld, first_bias, lam = None, 0, None, 0.0
    if first_values is not None:
        rows, column, bias_v, lam = first_values
        nv = n_kv_heads * value_dim
        if rows.shape[0] != n or rows.shape[1] < column + nv or rows.dtype != qkv.dtype or (bias_v is not None and bias_v.numel() != nv):
            raise KernelError("qk_norm_rope: the values to mix in must be rows of qkv's dtype with the values' columns")
        first, first_ld = _dev(rows, "first values") + column * rows.element_size(), rows.shape[1]
        first_bias = _dev(bias_v, "first values' bias", f32) if bias_v is not None else None
    _check(load("qk_norm_rope").ni_qk_norm_rope(
        _dev(qkv, "qkv") + col0 * qkv.element_size(), _code(qkv, "qkv"), _code(q_out, "q_out"), qkv.shape[1], _dev(bias, "bias", f32) if bias is not None else None,
        _dev(q_gain, "q_gain", f32) if q_gain is not None else None, _dev(k_gain, "k_gain", f32) if k_gain is not None else None,
        float(eps), _dev(positions, "positions", i32), _dev(seq_of_token, "seq_of_token", i32),
        _dev(block_table, "block_table", i32), block_table.shape[1], _dev(inv_freq, "inv_freq", f32), float(magnitude),
        _dev(q_out, "q_out"), _dev(k_pages, "k_pages") if write else None, _dev(v_pages, "v_pages") if write else None,
        n, n_heads, n_kv_heads, head_dim, value_dim, rotary_dim, page_size, 1 if head_unit else 0, float(coef),
        float(every), first, first_ld, first_bias, float(lam), _stream()), "qk_norm_rope")


LIGHTNING_MAX_DIM = 256      # the largest key size whose chunk buffers fit a block's shared memory


def lightning_max_chunks(n_tokens: int, n_seqs: int) -> int:
    """The size of lightning_recurrence's buffer in units of H dim vdim floats, for ``n_seqs`` requests with
    ``n_tokens`` tokens in all: two entries (its own sum, the state before it) for each of the most chunks they
    can be cut into."""
    return int(load("lightning").ni_lightning_max_chunks(int(n_tokens), int(n_seqs)))


def lightning_recurrence(proj, state, cu_q, slots, n_seqs, decay, n_heads, dim, vdim, out, max_q_len=None, buf=None,
                         activation: bool = True) -> None:
    """Linear attention with a decay per head over a step's tokens, request by request: with q, k [H, dim] and v
    [H, vdim] = silu of proj's columns (q | k | v | ...), S <- decay_h S + k v^T and out = S^T q, all float32;
    ``state`` float32 [slots, >= H dim vdim] holds every request's S and advances by the step's tokens; out float32
    [T, H vdim].  ``max_q_len``: the most tokens one request brings (None: as many as there are tokens); a step
    of single tokens is one launch, others run in chunks and need ``buf`` (float32, lightning_max_chunks(T, n_seqs)
    x H dim vdim entries; None: allocated here).  ``activation`` False: proj (float32) holds q, k and v themselves -
    nothing is activated (a caller that has prepared them, e.g. rotated queries and scaled keys)."""
    n = proj.shape[0]
    if not activation and proj.dtype != torch.float32:
        raise KernelError("lightning_recurrence: q, k, v that enter as they are must be float32")
    if proj.shape[1] < n_heads * (2 * dim + vdim) or out.shape != (n, n_heads * vdim) or decay.numel() != n_heads \
            or state.shape[1] < n_heads * dim * vdim:
        raise KernelError("lightning_recurrence: shapes do not agree")
    max_q_len = n if max_q_len is None else int(max_q_len)
    per_chunk = n_heads * dim * vdim
    chunks = 0
    if max_q_len > 1:
        chunks = lightning_max_chunks(n, n_seqs)
        if buf is None:
            buf = torch.empty(chunks * per_chunk, dtype=torch.float32, device=proj.device)
        elif buf.numel() < chunks * per_chunk:
            raise KernelError("lightning_recurrence: the chunk buffer is too small")
    _check(load("lightning").ni_lightning_recurrence(
        _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], _dev(state, "state", torch.float32), state.shape[1],
        _dev(cu_q, "cu_q", torch.int32), _dev(slots, "slots", torch.int32), _dev(decay, "decay", torch.float32),
        _dev(out, "out", torch.float32), n, n_seqs, max_q_len, _dev(buf, "buf", torch.float32) if chunks else None,
        chunks, n_heads, dim, vdim, 1 if activation else 0, _stream()), "lightning_recurrence")


def linear_attention_prepare(proj, positions, inv_freq, k_scale, qkv, n_heads, dim, vdim, rotary_dim) -> None:
    """qkv[t] = [rot(q) | rot(k) * k_scale | v] in float32 from proj [T, ld] (columns q (H dim) | k (H dim) | v (H vdim)
    | ...): the first ``rotary_dim`` dimensions of every head of q and k are rotated, dimension i paired with
    i + rotary_dim / 2, by the angle float(position) * inv_freq[i]; the values are copied."""
    n = proj.shape[0]
    cols = n_heads * (2 * dim + vdim)
    if proj.shape[1] < cols or tuple(qkv.shape) != (n, cols) or (rotary_dim > 0 and inv_freq.numel() != rotary_dim // 2):
        raise KernelError("linear_attention_prepare: shapes do not agree")
    _check(load("lightning").ni_linear_attention_prepare(
        _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], _dev(positions, "positions", torch.int32),
        _dev(inv_freq, "inv_freq", torch.float32), float(k_scale), _dev(qkv, "qkv", torch.float32), n, n_heads, dim, vdim,
        int(rotary_dim), _stream()), "linear_attention_prepare")


def retention_token_step(proj, state, cu_q, slots, n_seqs, decay, n_heads, dim, vdim, out, positions, inv_freq, rotary_dim,
                         k_scale) -> None:
    """A step in which every request brings ONE token, for a retention layer, in one launch: q and k of proj's columns
    (q | k | v | ...) are rotated (as linear_attention_prepare does) and k scaled, then S <- decay_h S + k v^T and
    out = S^T q as in lightning_recurrence with ``activation`` False."""
    n = proj.shape[0]
    if n != n_seqs or proj.shape[1] < n_heads * (2 * dim + vdim) or out.shape != (n, n_heads * vdim) or \
            decay.numel() != n_heads or state.shape[1] < n_heads * dim * vdim or (rotary_dim > 0 and inv_freq.numel() != rotary_dim // 2):
        raise KernelError("retention_token_step: shapes do not agree (one token per request)")
    _check(load("lightning").ni_retention_token_step(
        _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], _dev(state, "state", torch.float32), state.shape[1],
        _dev(cu_q, "cu_q", torch.int32), _dev(slots, "slots", torch.int32), _dev(decay, "decay", torch.float32),
        _dev(out, "out", torch.float32), n_seqs, n_heads, dim, vdim, _dev(positions, "positions", torch.int32),
        _dev(inv_freq, "inv_freq", torch.float32), int(rotary_dim), float(k_scale), _stream()), "retention_token_step")


def group_gated_norm(o, proj, col0, weight, eps, y, group: int, gate: str = "sigmoid", scale: float = 1.0) -> None:
    """y = scale * o / sqrt(mean over each group of ``group`` neighbouring columns of o^2 + eps) * weight * act(proj[:,
    col0 : col0 + N]); o float32 [T, N], weight float32 [N] or None (1), y [T, N] of proj's dtype; ``gate`` "sigmoid" or
    "silu"."""
    n, width = o.shape
    if y.shape != o.shape or y.dtype != proj.dtype or proj.shape[0] != n or group <= 0 or width % group or \
            (weight is not None and weight.numel() != width) or gate not in ("sigmoid", "silu"):
        raise KernelError("group_gated_norm: shapes, dtypes or the gate's kind do not agree")
    _check(load("lightning").ni_group_gated_norm(
        _dev(o, "o", torch.float32), _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], int(col0),
        _dev(weight, "weight", torch.float32) if weight is not None else None, float(eps), _dev(y, "y"), n, width // group,
        int(group), 1 if gate == "silu" else 0, float(scale), _stream()), "group_gated_norm")


def lightning_gated_norm(o, proj, col0, weight, eps, y) -> None:
    """y = o / sqrt(mean(o^2) + eps) * weight * sigmoid(proj[:, col0 : col0 + N]) row by row; o float32 [T, N], weight
    float32 [N], y [T, N] of proj's dtype."""
    n, width = o.shape
    if y.shape != o.shape or y.dtype != proj.dtype or weight.numel() != width or proj.shape[0] != n:
        raise KernelError("lightning_gated_norm: shapes or dtypes do not agree")
    _check(load("lightning").ni_lightning_gated_norm(
        _dev(o, "o", torch.float32), _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], int(col0),
        _dev(weight, "weight", torch.float32), float(eps), _dev(y, "y"), n, width, _stream()), "lightning_gated_norm")


class ResidualStreams:
    """The residual stream of a model that carries several of them side by side: ``x`` float32 [T, S, d], written from
    the first sublayer's end on; before that all streams equal the one row per token in ``base`` [T, d].  What the last
    sublayer left - its output and how the streams are made anew from it - stays pending (``leave``) and is applied by
    the pass that reads the streams for the next sublayer (``read``)."""

    def __init__(self, base: torch.Tensor, streams: int) -> None:
        self.base, self.streams = base, int(streams)
        self.x: Optional[torch.Tensor] = None
        self.pending = None

    def leave(self, y, mix: torch.Tensor, out: torch.Tensor) -> None:
        """``y``: float32 [T, d], or the RoutedRows of experts not yet summed.  mix [S, S] (from, to), out [S]."""
        if self.pending is not None:
            raise KernelError("residual streams: an output is pending already")
        self.pending = (y, mix, out)

    def read(self, coef, tanh_norm=None, out_dtype=torch.float32, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """sum_s coef[s] x_s (``coef`` None: the plain sum) of the streams after the pending update; with ``tanh_norm`` =
        (alpha, weight, bias) float32: tanh(alpha u) * weight + bias in ``out_dtype``, else u itself, float32.  ``rows``
        int32: those rows only, and the streams stay as they are."""
        t, d = self.base.shape
        n = t if rows is None else rows.numel()
        h = torch.empty(n, d, dtype=out_dtype if tanh_norm is not None else torch.float32, device=self.base.device)
        source, target = (self.base if self.x is None else None), self.x
        keep = rows is None and self.pending is not None
        if keep and target is None:
            target = torch.empty(t, self.streams, d, dtype=torch.float32, device=self.base.device)
        hyper_step(target, source, self.streams, self.pending, coef, tanh_norm, h, rows, keep)
        if keep:
            self.x, self.pending = target, None
        return h


class RoutedRows:
    """What a step's routed experts left, not yet summed: y[t] = sum_j weights[t, j] * z[row of pair (t, j)], pair (t, j)'s
    row being row_of_pair[t top + j], t top + j itself (``row_of_pair`` None), or t E + ids[t, j] (``all_experts`` = E)."""

    def __init__(self, z, ids, weights, row_of_pair, all_experts: int = 0) -> None:
        self.z, self.ids, self.weights, self.row_of_pair, self.all_experts = z, ids, weights, row_of_pair, int(all_experts)


def hyper_step(x, base, streams: int, pending, coef, tanh_norm, h, rows, write_back: bool) -> None:
    """One pass over residual streams (see ResidualStreams): apply ``pending`` = (y or RoutedRows, mix, out) or None,
    write the streams back if asked, read them with ``coef`` and norm the sum into h."""
    f32, i32 = torch.float32, torch.int32
    d = h.shape[1]
    s = int(streams)
    if (x is not None and tuple(x.shape[1:]) != (s, d)) or (base is not None and base.shape[1] != d) or \
            (coef is not None and coef.numel() != s) or (rows is not None and rows.numel() != h.shape[0]):
        raise KernelError("hyper_step: shapes do not agree")
    n_tokens = base.shape[0] if base is not None else x.shape[0]
    if rows is None and h.shape[0] != n_tokens:
        raise KernelError("hyper_step: one output row per token")
    kind, y, r = 0, None, None
    mix = out = None
    if pending is not None:
        y, mix, out = pending
        if mix.shape != (s, s) or out.numel() != s:
            raise KernelError("hyper_step: the mixing coefficients do not fit the streams")
        kind = 1
        if isinstance(y, RoutedRows):
            kind, r, y = 2, y, None
            if r.z.shape[1] != d or r.ids.shape[0] != n_tokens:
                raise KernelError("hyper_step: the experts' rows do not fit the streams")
        elif y.shape != (n_tokens, d):
            raise KernelError("hyper_step: the sublayer's output does not fit the streams")
    if tanh_norm is not None and (tanh_norm[0].numel() != 1 or tanh_norm[1].numel() != d or tanh_norm[2].numel() != d):
        raise KernelError("hyper_step: the norm has another width")
    act = _code(r.z, "z") if r is not None else _code(h, "h")
    if r is not None and tanh_norm is not None and r.z.dtype != h.dtype:
        raise KernelError("hyper_step: the experts' rows and the normed output must share one dtype")
    if tanh_norm is None and h.dtype != f32:
        raise KernelError("hyper_step: without a norm the output is float32")

    def opt(t, name, dtype):
        return _dev(t, name, dtype) if t is not None else None

    _check(load("hyper").ni_hyper_step(
        opt(x, "x", f32), opt(base, "base", f32), s, d, h.shape[0], 1 if write_back else 0, kind, opt(y, "y", f32),
        _dev(r.z, "z") if r is not None else None, act, opt(r.ids if r else None, "ids", i32), opt(r.weights if r else None, "weights", f32),
        opt(r.row_of_pair if r else None, "row_of_pair", i32), r.ids.shape[1] if r is not None else 0,
        r.all_experts if r is not None else 0, opt(mix, "mix", f32), opt(out, "out", f32), opt(coef, "coef", f32),
        *((opt(v, "norm", f32) for v in tanh_norm) if tanh_norm is not None else (None, None, None)), _dev(h, "h"),
        opt(rows, "rows", i32), _stream()), "hyper_step")


HYPER_MAX_STREAMS = 32      # what the kernel keeps of a column in registers (checked against the built library)


def tanh_norm(h, delta, alpha, weight, bias, out, rows=None) -> None:
    """Residual add fused with the norm tanh(alpha h) * weight + bias: as add_rmsnorm, h float32 [T, d], delta float32
    or None (added into h unless ``rows`` is given)."""
    one = _unit_coefficients(h.device) if delta is not None else None
    hyper_step(h.view(h.shape[0], 1, h.shape[1]), None, 1, (delta, one.view(1, 1), one) if delta is not None else None, None,
               (alpha, weight, bias), out, rows, delta is not None and rows is None)


_units: Dict[torch.device, torch.Tensor] = {}


def _unit_coefficients(device) -> torch.Tensor:
    t = _units.get(device)
    if t is None:
        t = _units[device] = torch.ones(1, dtype=torch.float32, device=device)
    return t


def difference_norm(a, out, lam: float, eps: float, factor: float, token_list=None) -> None:
    """out[t, h, :] = u / sqrt(mean(u^2) + eps) * factor with u = a[t, 2h, :] - lam * a[t, 2h + 1, :]; a float32
    [T, 2 H V] (two maps per head), out [T, H V]; ``token_list`` int32: those tokens only."""
    n = a.shape[0] if token_list is None else token_list.numel()
    if a.dim() != 3 or out.shape != (a.shape[0], (a.shape[1] // 2) * a.shape[2]) or a.shape[1] % 2:
        raise KernelError("difference_norm: a must be [T, 2 H, V] and out [T, H V]")
    _check(load("difference").ni_difference_norm(
        _dev(a, "a", torch.float32), _dev(out, "out"), _code(out, "out"),
        _dev(token_list, "token_list", torch.int32) if token_list is not None else None, n, a.shape[1] // 2, a.shape[2],
        float(lam), float(eps), float(factor), _stream()), "difference_norm")


MLSTM_MAX_DIM = 256      # the largest key size whose chunk buffers fit a block's shared memory


def mlstm_state_floats(n_heads: int, dim: int, vdim: int) -> int:
    """Floats of one request's state: per head a record (matrix, normaliser, padded to 4), then every head's maximum."""
    record = -(-(dim * vdim + dim) // 4) * 4
    return n_heads * record + -(-n_heads // 4) * 4


def mlstm_buffer_floats(n_tokens: int, n_seqs: int, n_heads: int, dim: int, vdim: int) -> int:
    """Floats of scratch that mlstm_chunk_step needs."""
    f = load("mlstm").ni_mlstm_buffer_floats
    f.restype, f.argtypes = _LL, [_I] * 5
    return int(f(n_tokens, n_seqs, n_heads, dim, vdim))


def _mlstm_check(proj, gates, bias_i, bias_f, state, weight, y, n_heads, dim, vdim, what) -> None:
    n = proj.shape[0]
    if proj.shape[1] < 2 * n_heads * (dim + vdim) or gates.shape[0] != n or bias_i.numel() != n_heads or bias_f.numel() != n_heads \
            or state.shape[1] != mlstm_state_floats(n_heads, dim, vdim) or weight.numel() != n_heads * vdim or y.shape != (n, n_heads * vdim):
        raise KernelError(f"{what}: shapes do not agree")


def mlstm_token_step(proj, gates, col_i, col_f, bias_i, bias_f, cap, state, cu_q, slots, n_seqs, q_scale, weight, eps, y,
                     n_heads, dim, vdim) -> None:
    """A step in which every request brings ONE token, for a matrix-memory layer, in one launch: gates, state update,
    read-out, the norm per head and the output gate.  proj float32 [n_seqs, ld] with columns q | k | v | gate | ...; gates
    float32 [n_seqs, ldg] (it may be proj), the input gates' logits in columns col_i .. col_i + H, the forget gates' in
    col_f .. col_f + H; state float32 [slots, mlstm_state_floats]; y [n_seqs, H vdim]."""
    _mlstm_check(proj, gates, bias_i, bias_f, state, weight, y, n_heads, dim, vdim, "mlstm_token_step")
    f32, i32 = torch.float32, torch.int32
    _check(load("mlstm").ni_mlstm_token_step(
        _dev(proj, "proj", f32), proj.shape[1], _dev(gates, "gates", f32), gates.shape[1], int(col_i), int(col_f),
        _dev(bias_i, "bias_i", f32), _dev(bias_f, "bias_f", f32), float(cap), _dev(state, "state", f32), state.shape[1],
        _dev(cu_q, "cu_q", i32), _dev(slots, "slots", i32), n_seqs, float(q_scale), _dev(weight, "weight", f32), float(eps),
        _dev(y, "y"), _code(y, "y"), n_heads, dim, vdim, _stream()), "mlstm_token_step")


def mlstm_chunk_step(proj, gates, col_i, col_f, bias_i, bias_f, cap, state, cu_q, slots, n_seqs, max_q_len, q_scale, weight,
                     eps, buf, out, y, n_heads, dim, vdim) -> None:
    """Any step of a matrix-memory layer, chunk by chunk; arguments as mlstm_token_step, proj in the activations' type
    (y's too), buf float32 with mlstm_buffer_floats(...) entries, out float32 [T, H vdim] scratch.  Where the read-out
    kernel has a head's whole values it norms and gates them itself; otherwise group_gated_norm follows."""
    n = proj.shape[0]
    _mlstm_check(proj, gates, bias_i, bias_f, state, weight, y, n_heads, dim, vdim, "mlstm_chunk_step")
    if out.shape != y.shape or y.dtype != proj.dtype:
        raise KernelError("mlstm_chunk_step: out and y must be [T, H vdim], y of proj's dtype")
    f32, i32 = torch.float32, torch.int32
    finished = ctypes.c_int(0)
    _check(load("mlstm").ni_mlstm_chunk_step(
        _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], _dev(gates, "gates", f32), gates.shape[1], int(col_i), int(col_f),
        _dev(bias_i, "bias_i", f32), _dev(bias_f, "bias_f", f32), float(cap), _dev(state, "state", f32), state.shape[1],
        _dev(cu_q, "cu_q", i32), _dev(slots, "slots", i32), n, n_seqs, int(max_q_len), float(q_scale),
        _dev(weight, "weight", f32), float(eps), _dev(buf, "buf", f32), buf.numel(), _dev(out, "out", f32), _dev(y, "y"),
        ctypes.byref(finished), n_heads, dim, vdim, _stream()), "mlstm_chunk_step")
    if not finished.value:
        group_gated_norm(out, proj, 2 * n_heads * dim + n_heads * vdim, weight, eps, y, vdim, gate="sigmoid")


def conv_qk_prepare(proj, conv_w, q_gain, k_gain, eps, state, positions, seq_of_token, cu_q, slots, n_seqs, block_table,
                    inv_freq, q_out, k_pages, v_pages, n_heads, n_kv_heads, head_dim, rotary_dim, taps, page_size) -> None:
    """From the fused projection ``proj`` [T, ld] (columns: the queries' channels, the keys' channels, then whatever
    else): causal convolution over time per channel (``conv_w`` float32 [taps, C] - tap-major -, the last tap the token's own;
    what lies before a portion comes from the request's history in ``state`` float32 [slots, (taps - 1) C]), RMS
    norm per head (``q_gain`` / ``k_gain`` float32 [head_dim]), rotation of adjacent pairs of the first
    ``rotary_dim`` dimensions; queries -> q_out [T, H hd], keys -> k_pages, the keys' convolution output as it is ->
    v_pages (pages [P, Hkv, page_size, hd]; None: nothing is written); then the history moves on."""
    n = proj.shape[0]
    c = (n_heads + n_kv_heads) * head_dim
    write = k_pages is not None
    f32, i32 = torch.float32, torch.int32
    if proj.shape[1] < c or q_out.shape != (n, n_heads * head_dim) or conv_w.shape != (taps, c):
        raise KernelError("conv_qk_prepare: shapes do not agree")
    if q_out.dtype != proj.dtype or (write and (k_pages.dtype != proj.dtype or v_pages.dtype != proj.dtype)):
        raise KernelError("conv_qk_prepare: all activations must share one dtype")
    if write and (tuple(k_pages.shape[1:]) != (n_kv_heads, page_size, head_dim) or v_pages.shape != k_pages.shape):
        raise KernelError("conv_qk_prepare: pages must be [P, Hkv, page_size, head_dim]")
    if state.shape[1] != (taps - 1) * c or q_gain.numel() != head_dim or k_gain.numel() != head_dim:
        raise KernelError("conv_qk_prepare: the state or a gain has another size")
    if rotary_dim > 0 and inv_freq.numel() != rotary_dim // 2:
        raise KernelError("conv_qk_prepare: inv_freq must have rotary_dim / 2 entries")
    _check(load("conv_attention").ni_conv_qk_prepare(
        _dev(proj, "proj"), _code(proj, "proj"), proj.shape[1], _dev(conv_w, "conv_w", f32), _dev(q_gain, "q_gain", f32),
        _dev(k_gain, "k_gain", f32), float(eps), _dev(state, "state", f32), state.shape[1],
        _dev(positions, "positions", i32), _dev(seq_of_token, "seq_of_token", i32), _dev(cu_q, "cu_q", i32),
        _dev(slots, "slots", i32), _dev(block_table, "block_table", i32), block_table.shape[1],
        _dev(inv_freq, "inv_freq", f32), _dev(q_out, "q_out"), _dev(k_pages, "k_pages") if write else None,
        _dev(v_pages, "v_pages") if write else None, n, n_seqs, n_heads, n_kv_heads, head_dim, rotary_dim, taps,
        page_size, _stream()), "conv_qk_prepare")


ROUTE_MAX_EXPERTS = 256      # what the routing kernel keeps in shared memory per token


def route(x, w_router, bias, ids, weights, counts, n_real, top, renormalize=False, sigmoid_scores=False,
          all_scores=None, groups: int = 1, keep_groups: int = 1, weight_scale: float = 1.0) -> None:
    """Per token: scores = softmax(w_router x), or with ``sigmoid_scores`` sigmoid(w_router x), each expert on its own
    (float32; w_router float32 [E, d]); ``all_scores`` float32 [T, n_real] (or None) receives every real expert's score;
    the ``top`` experts with the
    largest score + bias (``bias`` float32 [E] or None) -> ids int32 [T, top], their scores -> weights float32
    [T, top] (divided by their sum if ``renormalize``, then times ``weight_scale``).  ``groups`` > 1: the experts, in
    their order, are split into that many groups of one size, ranked by their best expert, and all but the first
    ``keep_groups`` drop out.  ``counts`` int32 [n_real] (or None) receives how many
    tokens chose each of the first ``n_real`` experts (added to what it holds)."""
    n, d = x.shape
    e = w_router.shape[0]
    if w_router.shape != (e, d) or ids.shape != (n, top) or weights.shape != (n, top) or (bias is not None and bias.numel() != e):
        raise KernelError("route: shapes do not agree")
    if e > ROUTE_MAX_EXPERTS:
        raise KernelError(f"route: {e} experts, more than the kernel's {ROUTE_MAX_EXPERTS}")
    _check(load("routed").ni_route(_dev(x, "x"), _code(x, "x"), _dev(w_router, "w_router", torch.float32),
                                   _dev(bias, "bias", torch.float32) if bias is not None else None,
                                   _dev(ids, "ids", torch.int32), _dev(weights, "weights", torch.float32),
                                   _dev(counts, "counts", torch.int32) if counts is not None else None, n, d, e, n_real, top,
                                   1 if renormalize else 0, 1 if sigmoid_scores else 0,
                                   _dev(all_scores, "all_scores", torch.float32) if all_scores is not None else None,
                                   int(groups), int(keep_groups), float(weight_scale), _stream()), "route")


def route_layout(ids, counts, offsets, tile_first, cursor, row_of_pair, token_of_row, n_real, weights=None,
                 weight_of_row=None) -> None:
    """Lay the (token, choice) pairs out expert by expert: offsets / tile_first int32 [n_real + 1] (first row and
    first 64-row tile of each expert's stretch), row_of_pair int32 [T top] (-1 for pairs of identity experts),
    token_of_row int32 [T top]; counts comes from route() and is left zero, cursor int32 [n_real] is scratch.
    With ``weights`` (route's) and ``weight_of_row`` float32 [T top], every row also receives its pair's weight."""
    n, top = ids.shape
    i32 = torch.int32
    if offsets.numel() < n_real + 1 or tile_first.numel() < n_real + 1 or row_of_pair.numel() < n * top or token_of_row.numel() < n * top:
        raise KernelError("route_layout: a buffer is too small")
    _check(load("routed").ni_route_layout(_dev(ids, "ids", i32), _dev(counts, "counts", i32), _dev(offsets, "offsets", i32),
                                          _dev(tile_first, "tile_first", i32), _dev(cursor, "cursor", i32),
                                          _dev(row_of_pair, "row_of_pair", i32), _dev(token_of_row, "token_of_row", i32),
                                          n * top, top, n_real,
                                          _dev(weights, "weights", torch.float32) if weight_of_row is not None else None,
                                          _dev(weight_of_row, "weight_of_row", torch.float32) if weight_of_row is not None else None,
                                          _stream()), "route_layout")


PLAIN_GLU = (float("inf"), 1.0, 0.0)      # (limit, slope, shift) of silu(gate) * up


NO_ACT, GATED_ACT, RELU2_ACT = 0, 1, 2     # what an expert's first product ends with


def expert_gemm(a, token_of_row, w, out, offsets, tile_first, n_pairs, act: int, glu=PLAIN_GLU, row_scale=None) -> None:
    """out[row] = a[row] . w[e]^T for the rows of every expert e's stretch (``token_of_row`` given: a[token of the
    row]); w [E, N, K] (``act`` RELU2_ACT: out = the square of the product's positive part), or with GATED_ACT [E, 2N, K]
    (gate rows, then up rows) and out = the gated unit's activation with ``glu`` = (limit, slope, shift) and ``row_scale`` float32 [rows] (see capped_glu; the default is silu(gate) *
    up).  Each output element is one ascending chain of FP32 fused multiply-adds."""
    e, wn, k = w.shape
    act = int(act)
    n = wn // 2 if act == GATED_ACT else wn
    if a.shape[1] != k or out.shape[1] != n or out.shape[0] < n_pairs or a.dtype != w.dtype or out.dtype != w.dtype:
        raise KernelError("expert_gemm: shapes or dtypes do not agree")
    _check(load("routed").ni_expert_gemm(_dev(a, "a"), _code(a, "a"),
                                         _dev(token_of_row, "token_of_row", torch.int32) if token_of_row is not None else None,
                                         _dev(w, "w"), _dev(out, "out"), _dev(offsets, "offsets", torch.int32),
                                         _dev(tile_first, "tile_first", torch.int32), n_pairs, e, n, k, act,
                                         float(glu[0]), float(glu[1]), float(glu[2]),
                                         _dev(row_scale, "row_scale", torch.float32) if row_scale is not None else None,
                                         _stream()), "expert_gemm")


EXPERT_ROWS_MAX_PAIRS = 64      # (token, choice) pairs up to which a step takes the kernel with one warp per output


def expert_rows(a, w, out, ids, gather: bool, act: int, glu=PLAIN_GLU, row_scale=None) -> None:
    """A few rows, bfloat16: out[p] = a[p or p / top] . w[ids[p]]^T for every pair p of a real expert (others are
    skipped), one warp per output; ``act`` as in expert_gemm.  K must be a multiple of 8."""
    e, wn, k = w.shape
    act = int(act)
    n = wn // 2 if act == GATED_ACT else wn
    n_pairs, top = ids.numel(), ids.shape[1]
    bf = torch.bfloat16
    if a.shape[1] != k or out.shape != (n_pairs, n) or a.shape[0] != (n_pairs // top if gather else n_pairs):
        raise KernelError("expert_rows: shapes do not agree")
    _check(load("routed").ni_expert_rows(_dev(a, "a", bf), _dev(w, "w", bf), _dev(out, "out", bf), _dev(ids, "ids", torch.int32),
                                         n_pairs, top, 1 if gather else 0, e, n, k, act,
                                         float(glu[0]), float(glu[1]), float(glu[2]),
                                         _dev(row_scale, "row_scale", torch.float32) if row_scale is not None else None,
                                         _stream()), "expert_rows")


def route_combine(z, x, ids, weights, row_of_pair, y, n_real, all_experts: int = 0, unit_real: bool = False,
                  accumulate: bool = False) -> None:
    """y[t] = sum_j weights[t, j] * (z[row of pair (t, j)] for a real expert, x[t] for an identity expert), in the
    order of the choices, float32; row_of_pair None: pair p's row is p; ``all_experts`` = E > 0: z holds a row
    for every (token, expert), [T E, d], and the pair's row is t E + its expert.  ``unit_real``: real experts' rows
    count with weight 1 (their weight went into their input); ``accumulate``: the sum is added to what y holds."""
    n, top = ids.shape
    d = x.shape[1]
    if y.shape != (n, d) or z.shape[1] != d or z.dtype != x.dtype:
        raise KernelError("route_combine: shapes or dtypes do not agree")
    _check(load("routed").ni_route_combine(_dev(z, "z"), _dev(x, "x"), _code(x, "x"), _dev(ids, "ids", torch.int32),
                                           _dev(weights, "weights", torch.float32),
                                           _dev(row_of_pair, "row_of_pair", torch.int32) if row_of_pair is not None else None,
                                           _dev(y, "y", torch.float32), n, d, top, n_real, int(all_experts),
                                           1 if unit_real else 0, 1 if accumulate else 0, _stream()),
           "route_combine")


def route_combine_add_normed(z, x, ids, weights, row_of_pair, h, gain, eps, n_real, all_experts: int = 0,
                             unit_real: bool = False) -> None:
    """h[t] += y / sqrt(mean(y^2) + eps) * gain with y the sum that route_combine computes; h float32 [T, d]."""
    n, top = ids.shape
    d = x.shape[1]
    if h.shape != (n, d) or z.shape[1] != d or z.dtype != x.dtype or gain.numel() != d:
        raise KernelError("route_combine_add_normed: shapes or dtypes do not agree")
    _check(load("routed").ni_route_combine_add_normed(
        _dev(z, "z"), _dev(x, "x"), _code(x, "x"), _dev(ids, "ids", torch.int32), _dev(weights, "weights", torch.float32),
        _dev(row_of_pair, "row_of_pair", torch.int32) if row_of_pair is not None else None, _dev(h, "h", torch.float32),
        _dev(gain, "gain", torch.float32), float(eps), n, d, top, n_real, int(all_experts), 1 if unit_real else 0,
        _stream()), "route_combine_add_normed")


GEMV_MAX_ROWS = 16      # what the skinny kernels take
# Up to this many rows the engine uses them.  With 9 to 16 rows they need two batch tiles, which
# halves the blocks per SM and the loads in flight: measured on a decode step at batch 16,
# 1.40 ms against 1.21 ms for the library product with separate element-wise kernels.
SKINNY_ROWS = 8
STORE_BF16, STORE_F32, ADD_F32, SWIGLU_BF16 = 0, 1, 2, 3
GEGLU_BF16 = SWIGLU_BF16 | 16      # as SWIGLU_BF16 with the tanh form of gelu for the gate (NI_MODE_GELU)


def _gemv_check(m: int, n: int, k: int, w: torch.Tensor, out: torch.Tensor, mode: int, what: str) -> None:
    if w.shape != (n, k):
        raise KernelError(f"{what}: shapes do not agree")
    if m > GEMV_MAX_ROWS or k % 8:
        raise KernelError(f"{what}: takes at most {GEMV_MAX_ROWS} rows and K a multiple of 8 "
                          f"(got M={m}, K={k})")
    if mode in (SWIGLU_BF16, GEGLU_BF16):
        if n % 16 or out.shape != (m, n // 2) or out.dtype != torch.bfloat16:
            raise KernelError(f"{what}: the SwiGLU epilogue needs N a multiple of 16 and out bf16 [M, N/2]")
    else:
        want = torch.bfloat16 if mode == STORE_BF16 else torch.float32
        if out.shape != (m, n) or out.dtype != want:
            raise KernelError(f"{what}: out must be {want} [M, N]")


def warm_region(warm) -> tuple:
    """(address, bytes) of a hint ``(tensor, first byte, bytes)`` - a stretch of a tensor that a
    kernel asks into L2 on its way - cut to the tensor and to multiples of 16 bytes; (None, 0) for None."""
    if warm is None:
        return None, 0
    t, first, nbytes = warm
    size = t.numel() * t.element_size()
    first = min(max(int(first), 0), size) & ~15
    nbytes = min(int(nbytes), size - first) & ~15
    if nbytes <= 0 or not t.is_cuda or (t.data_ptr() + first) % 16:
        return None, 0
    return t.data_ptr() + first, nbytes


HANDOFF_ROWS = 8      # rows up to which a norm can be handed from the kernel that adds into the stream to its reader


class NormHandoff:
    """A norm prepared by the kernel that last added into the residual stream, for the kernel that
    reads it (up to HANDOFF_ROWS rows): ``x`` = bfloat16(h * gain) [M, d], ``ssq`` float32
    [8, parts] = per row and tile of columns the sum of h^2 (parts: the tiles rounded up to a multiple
    of 4, the rest zero), ``eps``.  The reader multiplies its
    finished products by 1 / sqrt(sum(ssq) / d + eps) per row: together RMSNorm(h) * gain without a
    kernel of its own.  ``norm`` is the part it stands for."""

    def __init__(self, norm, gain: torch.Tensor, eps: float, rows: int, width: int, tiles: int, device) -> None:
        self.norm, self.gain, self.eps, self.tiles = norm, gain, float(eps), int(tiles)
        self.parts = -(-self.tiles // 4) * 4
        self.x = torch.empty(rows, width, dtype=torch.bfloat16, device=device)
        self.ssq = torch.empty(8, self.parts, dtype=torch.float32, device=device)
        if self.parts != self.tiles:
            self.ssq[:, self.tiles:].zero_()        # what no tile writes must add nothing

    def producer_args(self):
        return _dev(self.gain, "gain", torch.float32), self.x.data_ptr(), self.ssq.data_ptr(), self.parts

    def reader_args(self):
        return self.ssq.data_ptr(), self.parts, self.eps


class StreamCopy:
    """What a block may hand to the block after it instead of a pending addition: the stream is up to date, and
    ``rounded`` is its bfloat16 copy, written by the kernel that last added into the stream.  The model passes it on
    only to a block that says ``takes_stream_copy``."""

    def __init__(self, stream: torch.Tensor, rounded: torch.Tensor) -> None:
        self.stream, self.rounded = stream, rounded


_NO_HANDOFF = (None, None, None, 0)
_NO_PRE = (None, 0, 0.0)


def gemv_out_tiles(m: int, n: int, k: int) -> int:
    """How many tiles of output columns the skinny product that adds [m, n] into the stream works in
    (the partial sums per row of a NormHandoff) - of whichever kernel linear_bf16 picks - or 0 if that
    kernel cannot prepare a norm for these sizes."""
    if m <= KSPLIT_ROWS and KSPLIT_MIN_K <= k <= KSPLIT_MAX_K and gemv_ksplit_supports(m, n, k):
        return int(load("gemv_ksplit").ni_gemv_ksplit_out_tiles(n, k))
    lib = load("gemv_bf16")
    return int(lib.ni_gemv_bf16_out_tiles(n, ADD_F32)) if lib.ni_gemv_bf16_writes_handoff(m, n, k) else 0


def gemv_reads_handoff(m: int, k: int) -> bool:
    """True if the skinny products can take a prepared norm on an input of m rows and width k."""
    return bool(load("gemv_bf16").ni_gemv_bf16_reads_handoff(m, k))


def gemv_bf16(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, mode: int, warm=None,
              handoff: Optional["NormHandoff"] = None, pre: Optional["NormHandoff"] = None, affine=None) -> None:
    """x[M, K] . w[N, K]^T for M <= 16, K % 8 == 0.  mode STORE_BF16 / STORE_F32: out[M, N] =;
    ADD_F32: out[M, N] +=; SWIGLU_BF16: w's rows in blocks of 8 gate + 8 up rows,
    out[M, N/2] = silu(gate) * up (GEGLU_BF16: gelu).  ``affine`` (scale, shift), each float32 [N] or None, with ADD_F32:
    out[M, N] += product * scale + shift.  ``warm`` (tensor, first byte, bytes): weights of the kernels
    after this one, asked into L2 when this kernel's own loads have been issued.  ``handoff`` (with
    ADD_F32, up to 8 rows): also prepare the norm that follows; ``pre``: x is such a prepared input."""
    if (handoff is not None or pre is not None) and x.shape[0] > HANDOFF_ROWS:
        raise KernelError("gemv_bf16: a norm is handed over for at most 8 rows")
    if handoff is not None and (mode != ADD_F32 or handoff.x.shape != out.shape or handoff.tiles != int(load("gemv_bf16").ni_gemv_bf16_out_tiles(w.shape[0], ADD_F32))):
        raise KernelError("gemv_bf16: the handoff does not fit this product")
    m, k = x.shape
    n = w.shape[0]
    _gemv_check(m, n, k, w, out, mode, "gemv_bf16")
    _check(load("gemv_bf16").ni_gemv_bf16(_dev(x, "x", torch.bfloat16), _dev(w, "w", torch.bfloat16),
                                          _dev(out, "out"), m, n, k, mode, *warm_region(warm),
                                          *(handoff.producer_args() if handoff is not None else _NO_HANDOFF),
                                          *(pre.reader_args() if pre is not None else _NO_PRE),
                                          *_affine_args(affine, n), _stream()), "gemv_bf16")


def _affine_args(affine, n: int) -> tuple:
    """(scale, shift) of an adding product as pointers (null where absent)."""
    if affine is None:
        return None, None
    scale, shift = affine
    if any(v is not None and v.numel() != n for v in (scale, shift)):
        raise KernelError("an adding product's scale and shift must have one number per column")
    return _f32_or_none(scale, "scale"), _f32_or_none(shift, "shift")


KSPLIT_ROWS = 8          # rows the cluster split-K skinny product takes
# The engine uses it for 2,048 < K <= 8,192 (2 to 4 slices).  Measured at 8 rows, against gemv_bf16:
# N 2,048 x K 8,192: 8.5 us against 10.1;  3,072 x 8,192: 11.1 against 16.7;  4,096 x 4,096: 8.5 against 10.2;
# 3,072 x 3,072: 7.0 against 8.3;  but 4,096 x 14,336 (7 slices: 37 clusters of 7 blocks leave SMs idle): 27.8 against 26.4.
KSPLIT_MIN_K, KSPLIT_MAX_K = 2049, 8192


def gemv_ksplit_supports(m: int, n: int, k: int) -> bool:
    """True if gemv_ksplit takes the product: up to 8 rows, K a multiple of 8 in 2 to 8 slices of at most 2,048."""
    return bool(load("gemv_ksplit").ni_gemv_ksplit_supports(m, n, k))


def gemv_ksplit(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, mode: int, warm=None,
                handoff: Optional["NormHandoff"] = None, pre=None, affine=None) -> None:
    """x[M, K] . w[N, K]^T for M <= 8 and a long K, split over the blocks of a cluster (each keeps
    its slice of the activations in registers; the slices' sums are added in slice order).
    mode STORE_BF16 / STORE_F32 / ADD_F32 (with ``affine``) as gemv_bf16."""
    m, k = x.shape
    n = w.shape[0]
    if mode not in (STORE_BF16, STORE_F32, ADD_F32):
        raise KernelError("gemv_ksplit: mode must be STORE_BF16, STORE_F32 or ADD_F32")
    _gemv_check(m, n, k, w, out, mode, "gemv_ksplit")
    if not gemv_ksplit_supports(m, n, k):
        raise KernelError(f"gemv_ksplit: M={m}, N={n}, K={k} is not supported (up to 8 rows, K in 2 to 8 slices of 2,048)")
    if pre is not None:
        raise KernelError("gemv_ksplit: takes no prepared norm on its input")
    if handoff is not None and (mode != ADD_F32 or handoff.x.shape != out.shape
                                or handoff.tiles != int(load("gemv_ksplit").ni_gemv_ksplit_out_tiles(n, k))):
        raise KernelError("gemv_ksplit: the handoff does not fit this product")
    _check(load("gemv_ksplit").ni_gemv_ksplit(_dev(x, "x", torch.bfloat16), _dev(w, "w", torch.bfloat16),
                                              _dev(out, "out"), m, n, k, mode, *warm_region(warm),
                                              *(handoff.producer_args() if handoff is not None else _NO_HANDOFF),
                                              *_affine_args(affine, n), _stream()), "gemv_ksplit")


def gemv_norm_bf16(h: torch.Tensor, gain: torch.Tensor, eps: float, rows: Optional[torch.Tensor],
                   w: torch.Tensor, out: torch.Tensor, mode: int, warm=None) -> None:
    """The same product with RMSNorm fused in front: x = norm(h[rows]) * gain, h float32
    [*, K] (the residual stream), rows int32 [M] or None for rows 0..M-1.  (``warm`` is accepted
    and dropped: the kernels with the norm fused run at their register limit and carry no request code.)"""
    k = h.shape[1]
    m = h.shape[0] if rows is None else rows.numel()
    n = w.shape[0]
    _gemv_check(m, n, k, w, out, mode, "gemv_norm_bf16")
    if gain.numel() != k:
        raise KernelError("gemv_norm_bf16: gain must have K entries")
    _check(load("gemv_bf16").ni_gemv_norm_bf16(
        _dev(h, "h", torch.float32), _dev(gain, "gain", torch.float32), float(eps),
        _dev(rows, "rows", torch.int32) if rows is not None else None, _dev(w, "w", torch.bfloat16),
        _dev(out, "out"), m, n, k, mode, *warm_region(warm), _stream()), "gemv_norm_bf16")


def gemv_qkv_rope(x: torch.Tensor, gain: Optional[torch.Tensor], eps: float, w: torch.Tensor,
                  q_out: torch.Tensor, k_pages: Optional[torch.Tensor], v_pages: Optional[torch.Tensor],
                  positions: torch.Tensor, seq_of_token: torch.Tensor, block_table: torch.Tensor,
                  inv_freq: torch.Tensor, n_q_heads: int, n_kv_heads: int, head_dim: int, rotary_dim: int,
                  page_size: int, warm=None, pre: Optional["NormHandoff"] = None) -> None:
    """Fused QKV projection of at most 16 single tokens: optional RMSNorm in front (x float32
    residual stream and ``gain`` given) or bfloat16 activations (gain None); rotary encoding of
    adjacent pairs and the paged K/V write behind.  q -> q_out bf16 [M, Hq hd]."""
    m, k = x.shape
    n = (n_q_heads + 2 * n_kv_heads) * head_dim
    if w.shape != (n, k) or q_out.shape != (m, n_q_heads * head_dim):
        raise KernelError("gemv_qkv_rope: shapes do not agree")
    if m > GEMV_MAX_ROWS or k % 8 or head_dim % 16:
        raise KernelError("gemv_qkv_rope: at most 16 rows, K a multiple of 8, head_dim a multiple of 16")
    write = k_pages is not None
    if write and tuple(k_pages.shape[1:]) != (n_kv_heads, page_size, head_dim):
        raise KernelError("gemv_qkv_rope: pages must be [P, Hkv, page_size, head_dim]")
    _check(load("gemv_bf16").ni_gemv_qkv_rope(
        _dev(x, "x", torch.float32 if gain is not None else torch.bfloat16),
        _dev(gain, "gain", torch.float32) if gain is not None else None, float(eps),
        _dev(w, "w", torch.bfloat16), _dev(q_out, "q_out", torch.bfloat16),
        _dev(k_pages, "k_pages", torch.bfloat16) if write else None,
        _dev(v_pages, "v_pages", torch.bfloat16) if write else None,
        _dev(positions, "positions", torch.int32), _dev(seq_of_token, "seq_of_token", torch.int32),
        _dev(block_table, "block_table", torch.int32), block_table.shape[1],
        _dev(inv_freq, "inv_freq", torch.float32), m, k, n_q_heads, n_kv_heads, head_dim, rotary_dim,
        page_size, 1 if write else 0, *warm_region(warm), *(pre.reader_args() if pre is not None else _NO_PRE),
        _stream()), "gemv_qkv_rope")


def linear_bf16(x: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype,
                residual: Optional[torch.Tensor] = None, warm=None, handoff: Optional["NormHandoff"] = None,
                affine=None):
    """y = x . w^T for bfloat16 operands with FP32 accumulation.

    Up to SKINNY_ROWS rows (decode): the package's own bandwidth kernel; with ``residual`` (float32
    [M, N]) the product is added into it and None is returned.  More rows: a library matrix
    product (cuBLASLt through torch), as the reference's projections are cuBLAS calls
    (src/op/kernels/cuda/matmul_kernel.cu:76-86); the caller adds the result to the residual.
    ``affine`` (scale, shift), with ``residual``: what is added is y * scale + shift (float32 per column, either may be
    None); where the kernel cannot add it, a ScaledAddition is returned.
    """
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16:
        raise KernelError("linear_bf16: operands must be bfloat16")
    if not x.is_cuda or not w.is_cuda:
        raise KernelError("linear_bf16: operands must be CUDA tensors")
    m, k = x.shape
    if m <= SKINNY_ROWS and k % 8 == 0:
        # a long contraction: K split over a cluster, activations in registers (else re-read per row tile)
        product = gemv_ksplit if (m <= KSPLIT_ROWS and KSPLIT_MIN_K <= k <= KSPLIT_MAX_K
                                  and gemv_ksplit_supports(m, w.shape[0], k)) else gemv_bf16
        if residual is not None:
            product(x, w, residual, ADD_F32, warm, handoff=handoff, affine=affine)
            return None
        out = torch.empty(m, w.shape[0], dtype=out_dtype, device=x.device)
        product(x, w, out, STORE_BF16 if out_dtype == torch.bfloat16 else STORE_F32, warm)
        return out
    if handoff is not None:
        raise KernelError("linear_bf16: a norm can only be handed over by the skinny product (up to 8 rows)")
    y = torch.matmul(x, w.t()) if out_dtype == torch.bfloat16 else torch.mm(x, w.t(), out_dtype=torch.float32)
    return y if affine is None else ScaledAddition(y, *affine)


_error_words: Dict[torch.device, torch.Tensor] = {}

# What the codes in the error word stand for (each kernel writes its own when a bounded wait runs out).
DEVICE_ERROR_CODES = {
    1: "tensor-core product (gemm_tc / gemm_tc2): the loader gave up waiting for a free stage",
    2: "tensor-core product (gemm_tc / gemm_tc2): the MMA issuer gave up waiting",
    3: "tensor-core product (gemm_tc / gemm_tc2): the epilogue gave up waiting for an accumulator",
    11: "tensor-core prefill attention: the loader gave up waiting",
    12: "tensor-core prefill attention: the MMA issuer gave up waiting",
    13: "tensor-core prefill attention: the softmax warps gave up waiting",
    21: "swapped-operand product (gemm_swap_tc): the loader gave up waiting",
    22: "swapped-operand product (gemm_swap_tc): the MMA issuer gave up waiting",
    23: "swapped-operand product (gemm_swap_tc): the epilogue gave up waiting",
    31: "fused decode step (decode_fused): a grid barrier was not reached by every block in time",
    32: "fused decode step (decode_fused): the weight loader gave up waiting for a free stage",
    33: "fused decode step (decode_fused): a consumer gave up waiting for its weights",
    41: "delta rule in chunks (delta_chunk): the scan gave up waiting for a chunk's operands",
}


def error_word(device) -> torch.Tensor:
    """The device's error word: int32 [1], zero unless a kernel recorded that one of its bounded
    waits ran out.  The engine copies it to the host with every step's sampled ids."""
    device = torch.device(device)
    if device.index is None:
        device = torch.device(device.type, torch.cuda.current_device())
    w = _error_words.get(device)
    if w is None:
        w = _error_words[device] = torch.zeros(1, dtype=torch.int32, device=device)
    return w


_error_word = error_word


def describe_device_error(code: int) -> str:
    return f"code {code}: {DEVICE_ERROR_CODES.get(code, 'unknown kernel')}"


def check_device_errors(device=None) -> None:
    """Raise if a kernel recorded that one of its bounded waits ran out (synchronises), and
    clear the record."""
    for dev, w in _error_words.items():
        if device is not None and dev != torch.device(device):
            continue
        code = int(w.item())
        if code:
            w.zero_()
            raise KernelError(f"a kernel on {dev} gave up waiting ({describe_device_error(code)}); "
                              f"the results of that step are not valid")


_WAIT_SETTERS = {"gemm_tc": "ni_gemm_tc_set_wait", "gemm_tc2": "ni_gemm_tc2_set_wait",
                 "gemm_swap_tc": "ni_gemm_swap_tc_set_wait",
                 "attention_prefill_tc": "ni_attention_prefill_tc_set_wait", "delta_chunk": "ni_delta_chunk_set_wait"}


def set_wait_limit(module: str, ticks: int = 0, extra_wait: bool = False) -> None:
    """How long a wait inside the module's kernels may last, in clock ticks (0: the default of one
    to two seconds).  ``extra_wait`` makes the kernels wait once more at their end for something
    that never comes - the way the tests make a bounded wait run out."""
    if module not in _WAIT_SETTERS:
        raise KernelError(f"module '{module}' has no bounded waits to set")
    _check_plain(getattr(load(module), _WAIT_SETTERS[module])(int(ticks), 1 if extra_wait else 0),
                 f"set_wait_limit({module})")


def gemm_tc(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor, mode: int, kernel: Optional[str] = None,
            accumulators: int = 2, tile_n: int = 0) -> None:
    """out = a[M, K] . b[N, K]^T on the tcgen05 tensor cores (bfloat16 in, FP32 accumulate).
    mode STORE_BF16 / STORE_F32 / ADD_F32 as in gemv_bf16; SWIGLU_BF16: b's rows in blocks of 8
    gate + 8 up rows, out bf16 [M, N/2].  ``kernel``: "pair" = two SMs per 256 x 256 tile
    (gemm_tc2.cu; ``tile_n`` 128 / 192 / 256 columns per tile, 0 = chosen by size), "single" = one SM per
    128 x 256 tile (gemm_tc.cu); default: the pair kernel from 256 rows and 256 columns on."""
    m, k = a.shape
    n = b.shape[0]
    if b.shape[1] != k:
        raise KernelError("gemm_tc: inner sizes do not agree")
    if k % 8:
        raise KernelError(f"gemm_tc: K must be a multiple of 8 (got {k})")
    if mode in (SWIGLU_BF16, GEGLU_BF16):
        if n % 16 or out.shape != (m, n // 2) or out.dtype != torch.bfloat16:
            raise KernelError("gemm_tc: the SwiGLU epilogue needs N a multiple of 16 and out bf16 [M, N/2]")
    else:
        want = torch.bfloat16 if mode == STORE_BF16 else torch.float32
        if out.shape != (m, n) or out.dtype != want:
            raise KernelError(f"gemm_tc: out must be {want} [M, N]")
    if kernel is None:
        kernel = "pair" if (GEMM_PAIR_DEFAULT and m >= 256 and n >= 256) else "single"
    if kernel == "pair":
        _check(load("gemm_tc2").ni_gemm_tc2(_dev(a, "a", torch.bfloat16), _dev(b, "b", torch.bfloat16), _dev(out, "out"),
                                            m, n, k, mode, accumulators, tile_n, _error_word(a.device).data_ptr(), _stream()),
               "gemm_tc2")
        return
    _check(load("gemm_tc").ni_gemm_tc(_dev(a, "a", torch.bfloat16), _dev(b, "b", torch.bfloat16), _dev(out, "out"),
                                      m, n, k, mode, _error_word(a.device).data_ptr(), _stream()), "gemm_tc")


# Two SMs per tile from 256 rows and columns on: 100 us against 113 us on the gate/up projection of
# a 2,048-token prompt (a block takes in a third less per k-block).
GEMM_PAIR_DEFAULT = True


ROPE_KV = 4                 # gemm_swap_tc: rotary encoding + paged K/V write of a fused QKV projection
SWAP_MAX_ROWS = 128         # most activation rows of the swapped-operand tensor-core product


def gemm_swap_scratch(m: int, n: int, k: int) -> int:
    """FP32 words of scratch that gemm_swap_tc needs for this product (0: K is not split)."""
    f = load("gemm_swap_tc").ni_gemm_swap_tc_scratch
    f.restype = ctypes.c_longlong
    return int(f(m, n, k))


def gemm_swap_tc(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, mode: int, scratch=None, tickets=None,
                 rope=None) -> None:
    """out = x[M, K] . w[N, K]^T for up to SWAP_MAX_ROWS rows on the tcgen05 tensor cores with the
    weights on the tile's 128 lanes (bfloat16 in, FP32 accumulate).  mode: STORE_BF16 / STORE_F32 /
    ADD_F32 / SWIGLU_BF16 as in gemv_bf16, or ROPE_KV with ``rope`` = (positions, seq_of_token,
    block_table, inv_freq, k_pages, v_pages, n_q_heads, n_kv_heads, head_dim, rotary_dim, page_size)
    and out = q [M, Hq * hd].  ``scratch`` (FP32, gemm_swap_scratch words) and ``tickets`` (int32
    zeros, one per 128 weight rows; left zero) are needed when K is split."""
    m, k = x.shape
    n = w.shape[0]
    if m > SWAP_MAX_ROWS or k % 8:
        raise KernelError(f"gemm_swap_tc: takes at most {SWAP_MAX_ROWS} rows and K a multiple of 8 (M={m}, K={k})")
    if w.shape[1] != k:
        raise KernelError("gemm_swap_tc: inner sizes differ")
    need = gemm_swap_scratch(m, n, k)
    if need and (scratch is None or tickets is None or scratch.numel() < need or tickets.numel() < -(-n // 128)):
        raise KernelError("gemm_swap_tc: scratch or tickets missing or too small")
    if mode == ROPE_KV:
        pos, seq, table, inv_freq, kp, vp, nq, nkv, hd, rot, page = rope
        extra = (_dev(pos, "positions", torch.int32), _dev(seq, "seq_of_token", torch.int32),
                 _dev(table, "block_table", torch.int32), table.shape[1], _dev(inv_freq, "inv_freq", torch.float32),
                 _dev(kp, "k_pages", torch.bfloat16) if kp is not None else None,
                 _dev(vp, "v_pages", torch.bfloat16) if vp is not None else None, nq, nkv, hd, rot, page)
        if out.shape != (m, nq * hd) or out.dtype != torch.bfloat16:
            raise KernelError("gemm_swap_tc: with ROPE_KV out is q, bfloat16 [M, Hq * hd]")
    else:
        extra = (None, None, None, 0, None, None, None, 0, 0, 0, 0, 0)
        want = (m, n // 2) if mode == SWIGLU_BF16 else (m, n)
        dt = torch.float32 if mode in (STORE_F32, ADD_F32) else torch.bfloat16
        if tuple(out.shape) != want or out.dtype != dt:
            raise KernelError(f"gemm_swap_tc: out must be {dt} {list(want)}")
    _check(load("gemm_swap_tc").ni_gemm_swap_tc(
        _dev(x, "x", torch.bfloat16), _dev(w, "w", torch.bfloat16), _dev(out, "out"), m, n, k, mode,
        _dev(scratch, "scratch", torch.float32) if need else None,
        _dev(tickets, "tickets", torch.int32) if need else None, *extra,
        _error_word(x.device).data_ptr(), _stream()), "gemm_swap_tc")


DECODE_HEAD_DIMS = (64, 128)
DECODE_SEGMENT_KEYS = {64: 64, 128: 64}      # keys per shared-memory buffer of a decode-attention block
DECODE_BLOCKS_PER_SM = 4
# The decode kernel reads all but a token's last DECODE_FRESH_KEYS keys while the kernel that
# writes this step's keys may still run, so a portion sent to it has at most this many tokens
# (the same constant as in attention_decode.cu; ni_attention_decode_fresh_keys() returns it).
DECODE_FRESH_KEYS = 2


def decode_splits(n_items: int, n_kv_heads: int, head_dim: int, max_kv_len: int, n_sms: Optional[int] = None) -> int:
    """How many blocks share one (token, kv head): as many as fill the GPU once (three blocks of
    the split kernel are resident per SM; a second wave costs more than longer blocks), each with
    at least 384 keys of the longest context - 256 when there are few pairs, whose blocks are
    bound by latency, not by bandwidth - and cut so that no block is left with a short remainder.
    Middle batches of 64-wide heads (more than one pair per SM): two or three lean blocks per pair,
    four of which fit an SM (batch 32 at 3,072 tokens: 48.1 us unsplit, 43.0 us in two).
    More pairs than the GPU holds at once: one lean block per pair with heads of 64 (four of
    those fit an SM); with heads of 128 (three per SM) the count, up to 4, that fills the last
    wave best (512 pairs: 58 % of two waves unsplit, 87 % of four waves in three parts)."""
    if n_sms is None:
        n_sms = sm_count()
    pairs = max(1, n_items * n_kv_heads)
    chunks = -(-max_kv_len // 64)                 # the kernel cuts a context into 64-key chunks
    slots = n_sms * 3
    if head_dim > 64 and pairs > slots:
        best, best_fill = 1, 0.0
        for s in range(1, 5):
            if s > 1 and chunks < 6 * s:
                break
            fill = pairs * s / (-(-pairs * s // slots) * slots)
            if fill > best_fill + 0.03:
                best, best_fill = s, fill
        per_split = -(-chunks // best)
        return max(1, -(-chunks // per_split))
    if (n_sms * DECODE_BLOCKS_PER_SM) // pairs <= 1:
        return 1                                  # large batch: one lean block per pair
    if pairs > n_sms and head_dim <= 64:          # more than one pair per SM: lean blocks, four per SM
        slots = n_sms * DECODE_BLOCKS_PER_SM
    fill = slots // pairs
    keys_per_split = 256 if pairs <= 16 else 384
    target = max(1, min(64, fill, -(-max_kv_len // keys_per_split)))
    per_split = -(-chunks // target)
    return max(1, -(-chunks // per_split))


PREFILL_MAX_HEAD_DIM = 128
PREFILL_TILE_ROWS = 128      # query rows per block of the flash-style kernel


DECODE_BALANCED_MAX_ITEMS = 1024


def attention_decode_balanced_scratch(n_q_heads: int, n_kv_heads: int, head_dim: int) -> int:
    """Scratch floats that attention_decode_balanced needs (two slots per block; independent of the batch)."""
    lib = load("attention_decode")
    lib.ni_attention_decode_balanced_scratch.restype = ctypes.c_longlong
    lib.ni_attention_decode_balanced_scratch.argtypes = [_I, _I, _I]
    return int(lib.ni_attention_decode_balanced_scratch(n_q_heads, n_kv_heads, head_dim))


def attention_decode_balanced(q, k_pages, v_pages, out, token_list, n_items, positions, seq_of_token, block_table,
                              n_q_heads, n_kv_heads, head_dim, page_size, window, scale, scratch, tickets, warm=()) -> None:
    """Attention of single query tokens (bfloat16) with the keys of all tokens dealt evenly over a fixed
    set of blocks (three per SM): for many tokens, or tokens of very different context lengths.
    scratch: float32, at least attention_decode_balanced_scratch(...); tickets: int32 zeros, at least
    n_items * Hkv (left zero by the kernel).  At most DECODE_BALANCED_MAX_ITEMS tokens.  ``warm`` as in
    attention_decode."""
    regions = [v for w_ in (list(warm) + [None, None])[:2] for v in warm_region(w_)]
    if head_dim not in DECODE_HEAD_DIMS or n_q_heads // n_kv_heads > 16 or n_items > DECODE_BALANCED_MAX_ITEMS:
        raise KernelError(f"attention_decode_balanced: head_dim {head_dim} / group {n_q_heads // n_kv_heads} / "
                          f"{n_items} tokens not supported")
    if scratch.numel() < attention_decode_balanced_scratch(n_q_heads, n_kv_heads, head_dim) or tickets.numel() < n_items * n_kv_heads:
        raise KernelError("attention_decode_balanced: scratch or tickets too small")
    _check(load("attention_decode").ni_attention_decode_balanced(
        _dev(q, "q", torch.bfloat16), _dev(k_pages, "k_pages", torch.bfloat16),
        _dev(v_pages, "v_pages", torch.bfloat16), _dev(out, "out", torch.bfloat16),
        _dev(token_list, "token_list", torch.int32) if token_list is not None else None, n_items,
        _dev(positions, "positions", torch.int32), _dev(seq_of_token, "seq_of_token", torch.int32),
        _dev(block_table, "block_table", torch.int32), block_table.shape[1], n_q_heads, n_kv_heads,
        head_dim, page_size, int(window) if window else 0, float(scale),
        _dev(scratch, "scratch", torch.float32), _dev(tickets, "tickets", torch.int32), *regions, _stream()),
        "attention_decode_balanced")


def attention_decode_cluster_merge(on: bool) -> None:
    """Whether the splits of a (token, kv head) merge inside a thread-block cluster where they can
    (the default) or always through the scratch buffer and the tickets."""
    _check_plain(load("attention_decode").ni_attention_decode_set_cluster_merge(1 if on else 0), "attention_decode")


def attention_decode(q, k_pages, v_pages, out, token_list, n_items, positions, seq_of_token, block_table,
                     n_q_heads, n_kv_heads, head_dim, page_size, window, scale, n_splits, scratch,
                     tickets, warm=(), score_cap: float = 0.0, chunk: int = 0, sink=None,
                     shared_pages: bool = False) -> None:
    """Split-K attention of single query tokens (bfloat16).  ``score_cap`` c > 0 bounds the scaled scores:
    s <- c * tanh(s / c).  ``chunk`` c > 0: the token at position p sees only the keys from p - p % c on; ``sink``
    float32 [Hq] (or True for zeros): exp(sink[h]) is added to head h's softmax denominator.  ``shared_pages``: the pages hold ONE head that all ``n_kv_heads`` of the
    call read (more than 16 query heads over one shared head, dealt over groups of at most 16).  ``token_list`` int32 [n_items] or
    None for tokens 0..n_items-1.  scratch: float32, at least n_items * Hq * n_splits *
    (head_dim + 2); tickets: int32 zeros, at least n_items * Hkv (left zero by the kernel).
    ``warm``: up to two (tensor, first byte, bytes) (weights that the kernels after it read): the
    kernel asks the first stretch into L2 when it starts, the second when its own stream has ended."""
    regions = [v for w_ in (list(warm) + [None, None])[:2] for v in warm_region(w_)]
    if head_dim not in DECODE_HEAD_DIMS or n_q_heads // n_kv_heads > 16:
        raise KernelError(f"attention_decode: head_dim {head_dim} / group {n_q_heads // n_kv_heads} not supported")
    if scratch.numel() < n_items * n_q_heads * n_splits * (head_dim + 2) or tickets.numel() < n_items * n_kv_heads:
        raise KernelError("attention_decode: scratch or tickets too small")
    lib = load("attention_decode")
    capped = score_cap and score_cap > 0.0
    if shared_pages and k_pages.shape[1] != 1:
        raise KernelError("attention_decode: shared pages hold one head")
    sink = _sinks(sink, n_q_heads, q.device)
    if chunk or sink is not None or shared_pages:
        _check(lib.ni_attention_decode_masked(
            _dev(q, "q", torch.bfloat16), _dev(k_pages, "k_pages", torch.bfloat16),
            _dev(v_pages, "v_pages", torch.bfloat16), _dev(out, "out", torch.bfloat16),
            _dev(token_list, "token_list", torch.int32) if token_list is not None else None, n_items,
            _dev(positions, "positions", torch.int32), _dev(seq_of_token, "seq_of_token", torch.int32),
            _dev(block_table, "block_table", torch.int32), block_table.shape[1], n_q_heads, n_kv_heads,
            head_dim, page_size, int(window) if window else 0, float(scale), float(score_cap or 0.0), int(chunk or 0),
            _f32_or_none(sink, "sink"), n_kv_heads if shared_pages else 0, n_splits, _dev(scratch, "scratch", torch.float32),
            _dev(tickets, "tickets", torch.int32),
            *regions, _stream()), "attention_decode")
        return
    _check((lib.ni_attention_decode_capped if capped else lib.ni_attention_decode)(
        _dev(q, "q", torch.bfloat16), _dev(k_pages, "k_pages", torch.bfloat16),
        _dev(v_pages, "v_pages", torch.bfloat16), _dev(out, "out", torch.bfloat16),
        _dev(token_list, "token_list", torch.int32) if token_list is not None else None, n_items,
        _dev(positions, "positions", torch.int32), _dev(seq_of_token, "seq_of_token", torch.int32),
        _dev(block_table, "block_table", torch.int32), block_table.shape[1], n_q_heads, n_kv_heads,
        head_dim, page_size, int(window) if window else 0, float(scale), *((float(score_cap),) if capped else ()), n_splits,
        _dev(scratch, "scratch", torch.float32), _dev(tickets, "tickets", torch.int32),
        *regions, _stream()), "attention_decode")


def attention_decode_difference(q, k_pages, v_pages, out, token_list, n_items, positions, seq_of_token, block_table, n_heads,
                                n_kv_heads, head_dim, page_size, scale, lam, eps, factor, n_splits, scratch, tickets, share: int = 1,
                                warm=()) -> None:
    """Split-K differential attention of single query tokens (bfloat16): every head has two maps.  q [T, H head_dim] (a
    head's two half rows one after the other); key pages [P, Hkv / share, page_size, head_dim] with the two maps side by
    side, value pages of the same shape; out [T, H head_dim] = (a_1 - lam a_2) / sqrt(mean(.^2) + eps) * factor per head.
    At most 8 heads per kv head; ``share`` > 1: that many neighbouring kv heads of the call read one head of the pages.
    The rest as attention_decode, with 2 H rows."""
    regions = [v for w_ in (list(warm) + [None, None])[:2] for v in warm_region(w_)]
    rows = 2 * n_heads // n_kv_heads
    if head_dim not in DECODE_HEAD_DIMS or rows > 16 or n_heads % n_kv_heads or n_kv_heads % share:
        raise KernelError(f"attention_decode_difference: head_dim {head_dim} / {rows} map rows per kv head not supported")
    if q.shape[1] != n_heads * head_dim or out.shape[1] != n_heads * head_dim or k_pages.shape[1] != n_kv_heads // share \
            or k_pages.shape[-1] != head_dim or v_pages.shape != k_pages.shape:
        raise KernelError("attention_decode_difference: shapes do not agree")
    if scratch.numel() < n_items * 2 * n_heads * n_splits * (head_dim + 2) or tickets.numel() < n_items * n_kv_heads:
        raise KernelError("attention_decode_difference: scratch or tickets too small")
    bf = torch.bfloat16
    _check(load("attention_decode").ni_attention_decode_difference(
        _dev(q, "q", bf), _dev(k_pages, "k_pages", bf), _dev(v_pages, "v_pages", bf), _dev(out, "out", bf),
        _dev(token_list, "token_list", torch.int32) if token_list is not None else None, n_items,
        _dev(positions, "positions", torch.int32), _dev(seq_of_token, "seq_of_token", torch.int32),
        _dev(block_table, "block_table", torch.int32), block_table.shape[1], 2 * n_heads, n_kv_heads, head_dim, page_size,
        float(scale), float(lam), float(eps), float(factor), int(share), n_splits, _dev(scratch, "scratch", torch.float32),
        _dev(tickets, "tickets", torch.int32), *regions, _stream()), "attention_decode_difference")


def attention_difference_tc_supports(head_dim: int, page_size: int) -> bool:
    """True if the tcgen05 differential attention takes the case: cached heads of 64 or 128, a page size from 8 to 128
    that divides 128."""
    return head_dim in (64, 128) and 8 <= page_size <= 128 and 128 % page_size == 0


def attention_prefill_difference(q, k_pages, v_pages, out, tile_seq, tile_row0, n_tiles, cu_q, kv_len, block_table, n_heads,
                                 n_kv_heads, head_dim, page_size, scale, lam, eps, factor) -> None:
    """Differential attention of prompt portions (bfloat16, tcgen05): operands as attention_decode_difference, tiles as
    attention_prefill; one block per tile and head runs the head's two maps as its two streams."""
    if not attention_difference_tc_supports(head_dim, page_size) or n_heads % n_kv_heads:
        raise KernelError(f"attention_prefill_difference: head_dim {head_dim} / page size {page_size} not supported")
    if q.shape[1] != n_heads * head_dim or out.shape != q.shape or tuple(k_pages.shape[1:]) != (n_kv_heads, page_size, head_dim) \
            or v_pages.shape != k_pages.shape:
        raise KernelError("attention_prefill_difference: shapes do not agree")
    bf, i32 = torch.bfloat16, torch.int32
    _check(load("attention_prefill_tc").ni_attention_prefill_tc_difference(
        _dev(q, "q", bf), _dev(k_pages, "k_pages", bf), _dev(v_pages, "v_pages", bf), _dev(out, "out", bf), q.shape[0],
        k_pages.shape[0], _dev(tile_seq, "tile_seq", i32), _dev(tile_row0, "tile_row0", i32), n_tiles, _dev(cu_q, "cu_q", i32),
        _dev(kv_len, "kv_len", i32), _dev(block_table, "block_table", i32), block_table.shape[1], n_heads, n_kv_heads, head_dim,
        page_size, float(scale), float(lam), float(eps), float(factor), _error_word(q.device).data_ptr(), _stream()),
        "attention_prefill_difference")


def attention_prefill_tc_supports(n_q_heads: int, n_kv_heads: int, head_dim: int, page_size: int) -> bool:
    """True if the tcgen05 prefill attention takes the case: head size 64 or 128, at least two
    query heads per kv head (an odd group's last head shares its block with a silent copy of
    itself), a page size from 8 to 128 that divides 128."""
    return (n_kv_heads > 0 and n_q_heads % n_kv_heads == 0 and n_q_heads // n_kv_heads >= 2
            and head_dim in (64, 128) and 8 <= page_size <= 128 and 128 % page_size == 0)


def attention_prefill(q, k_pages, v_pages, out, tile_seq, tile_row0, n_tiles, cu_q, kv_len, block_table,
                      n_q_heads, n_kv_heads, head_dim, page_size, window, scale, kernel: Optional[str] = None,
                      score_cap: float = 0.0, chunk: int = 0, sink=None) -> None:
    """``score_cap`` c > 0 bounds the scaled scores, s <- c * tanh(s / c) (the mma.sync kernel only).  ``chunk`` c > 0:
    a query at position p sees only the keys from p - p % c on; ``sink`` float32 [Hq] (or True for zeros): exp(sink[h]) is
    added to head h's softmax denominator (both kernels).
    Flash-style causal attention of prompt portions (bfloat16): one block per tile of
    PREFILL_TILE_ROWS query rows and query head (mma.sync kernel) or pair of query heads
    (tcgen05 kernel, where it takes the case); tile_seq / tile_row0 int32 [n_tiles] name each
    tile's request and first row.  ``kernel``: "tc" or "mma" to insist on one of the two."""
    if head_dim % 16 or head_dim > PREFILL_MAX_HEAD_DIM:
        raise KernelError(f"attention_prefill: head_dim {head_dim} not supported (multiples of 16 up to 128)")
    tc_ok = attention_prefill_tc_supports(n_q_heads, n_kv_heads, head_dim, page_size) and not score_cap
    sink = _sinks(sink, n_q_heads, q.device)
    if kernel == "tc" and not tc_ok:
        raise KernelError("attention_prefill: the tcgen05 kernel does not take this case")
    if tc_ok and kernel != "mma":
        _check(load("attention_prefill_tc").ni_attention_prefill_tc_masked(
            _dev(q, "q", torch.bfloat16), _dev(k_pages, "k_pages", torch.bfloat16),
            _dev(v_pages, "v_pages", torch.bfloat16), _dev(out, "out", torch.bfloat16), q.shape[0], k_pages.shape[0],
            _dev(tile_seq, "tile_seq", torch.int32), _dev(tile_row0, "tile_row0", torch.int32), n_tiles,
            _dev(cu_q, "cu_q", torch.int32), _dev(kv_len, "kv_len", torch.int32),
            _dev(block_table, "block_table", torch.int32), block_table.shape[1], n_q_heads, n_kv_heads,
            head_dim, page_size, int(window) if window else 0, float(scale), int(chunk or 0), _f32_or_none(sink, "sink"),
            _error_word(q.device).data_ptr(), _stream()), "attention_prefill_tc")
        return
    _check(load("attention_prefill").ni_attention_prefill(
        _dev(q, "q", torch.bfloat16), _dev(k_pages, "k_pages", torch.bfloat16),
        _dev(v_pages, "v_pages", torch.bfloat16), _dev(out, "out", torch.bfloat16),
        _dev(tile_seq, "tile_seq", torch.int32), _dev(tile_row0, "tile_row0", torch.int32), n_tiles,
        _dev(cu_q, "cu_q", torch.int32), _dev(kv_len, "kv_len", torch.int32),
        _dev(block_table, "block_table", torch.int32), block_table.shape[1], n_q_heads, n_kv_heads,
        head_dim, page_size, int(window) if window else 0, float(scale), float(score_cap or 0.0), int(chunk or 0),
        _f32_or_none(sink, "sink"), _stream()), "attention_prefill")


_argmax_keys: Dict[torch.device, torch.Tensor] = {}   # per device: merge keys, zero between calls


def argmax(logits: torch.Tensor, out: torch.Tensor) -> None:
    """out[r] = index of the largest logit of row r, ties to the lowest index."""
    n, v = logits.shape
    keys = _argmax_keys.get(logits.device)
    if keys is None and not torch.cuda.is_current_stream_capturing():
        keys = _argmax_keys[logits.device] = torch.zeros(4096, dtype=torch.int64, device=logits.device)
    use_keys = keys is not None and n <= keys.numel()
    _check(load("sampling").ni_argmax(_dev(logits, "logits", torch.float32), _dev(out, "out", torch.int32),
                                      n, v, keys.data_ptr() if use_keys else None, _stream()), "argmax")


def repetition_penalty(logits: torch.Tensor, ids: torch.Tensor, penalties: torch.Tensor) -> None:
    """In place: logits[r, id] = l / p if l > 0 else l * p for the ids listed in row r of
    ``ids`` (int32 [R, W], padded with -1, each id at most once per row)."""
    n, v = logits.shape
    if ids.shape[0] != n or penalties.numel() != n:
        raise KernelError("repetition_penalty: one id list and one penalty per row")
    _check(load("sampling").ni_repetition_penalty(
        _dev(logits, "logits", torch.float32), _dev(ids, "ids", torch.int32),
        _dev(penalties, "penalties", torch.float32), n, v, ids.shape[1], _stream()), "repetition_penalty")


def sample_by_cluster(on: bool) -> None:
    """Whether ``sample`` gives every row a thread-block cluster where the vocabulary allows it (the
    default) or always one block (the two give the same tokens; for comparisons)."""
    _check_plain(load("sampling").ni_sample_set_cluster(1 if on else 0), "sample")


def sample(logits, out, temperatures, top_ks, top_ps, seeds, counters) -> None:
    """One token per row by the row's own parameters; seeds and counters are 64-bit."""
    n, v = logits.shape
    for name, t in (("temperatures", temperatures), ("top_ks", top_ks), ("top_ps", top_ps),
                    ("seeds", seeds), ("counters", counters)):
        if t.numel() != n:
            raise KernelError(f"sample: {name} must have one entry per row")
    _check(load("sampling").ni_sample(
        _dev(logits, "logits", torch.float32), _dev(out, "out", torch.int32),
        _dev(temperatures, "temperatures", torch.float32), _dev(top_ks, "top_ks", torch.int32),
        _dev(top_ps, "top_ps", torch.float32), _dev(seeds, "seeds", torch.int64),
        _dev(counters, "counters", torch.int64), n, v, _stream()), "sample")


# ---- the fused decode step ---------------------------------------------------------------------------
FUSED_MAX_GROUPS = 4


class FusedLayer(ctypes.Structure):
    """One scheduled layer run of the fused decode kernel (mirrors FdLayer of decode_fused.cu)."""
    _fields_ = [("w_qkv", _P), ("w_o", _P), ("w_gate_up", _P), ("w_down", _P), ("gain_mixer", _P), ("gain_ffn", _P),
                ("k_pages", _P), ("v_pages", _P), ("eps_mixer", _F), ("eps_ffn", _F), ("write_cache", _I), ("group", _I)]


class FusedParams(ctypes.Structure):
    """Arguments of the fused decode kernel (mirrors FdParams of decode_fused.cu)."""
    _fields_ = [("layers", _P), ("inv_freq", _P), ("embedding", _P), ("lm_head", _P), ("gain_final", _P),
                ("tokens", _P), ("positions", _P), ("seq_of_token", _P), ("logit_rows", _P),
                ("tables", _P * FUSED_MAX_GROUPS),
                ("h", _P), ("q", _P), ("att", _P), ("act", _P), ("logits", _P), ("partials", _P), ("tickets", _P),
                ("barrier", _P), ("error", _P), ("trace", _P), ("wait_limit", _LL), ("bt_stride", _I * FUSED_MAX_GROUPS),
                ("n_layers", _I), ("M", _I), ("R", _I), ("d", _I), ("n_q_heads", _I), ("n_kv_heads", _I),
                ("head_dim", _I), ("rotary_dim", _I), ("inter", _I), ("vocab", _I), ("page_size", _I), ("window", _I),
                ("scale_log2e", _F), ("eps_final", _F), ("skip_arrive_at", _I)]


def decode_fused_lib() -> ctypes.CDLL:
    lib = load("decode_fused")
    if not getattr(lib, "_ni_checked", False):
        for fn, size in (("ni_decode_fused_params_size", ctypes.sizeof(FusedParams)),
                         ("ni_decode_fused_layer_size", ctypes.sizeof(FusedLayer))):
            f = getattr(lib, fn)
            f.restype = ctypes.c_longlong
            if int(f()) != size:
                raise KernelError(f"decode_fused: the argument records of the built kernel and of ops.py differ ({fn})")
        if lib.ni_decode_fused_max_groups() != FUSED_MAX_GROUPS:
            raise KernelError("decode_fused: FD_MAX_GROUPS of the built kernel differs from ops.FUSED_MAX_GROUPS")
        lib._ni_checked = True
    return lib


def decode_fused_supports(m: int, d: int, n_q_heads: int, n_kv_heads: int, head_dim: int, rotary_dim: int,
                          inter: int, vocab: int, page_size: int) -> bool:
    return bool(decode_fused_lib().ni_decode_fused_supports(m, d, n_q_heads, n_kv_heads, head_dim, rotary_dim, inter,
                                                            vocab, page_size))


def decode_fused_partials(m: int, n_kv_heads: int, head_dim: int) -> int:
    f = decode_fused_lib().ni_decode_fused_partials
    f.restype = ctypes.c_longlong
    f.argtypes = [_I, _I, _I]
    return int(f(m, n_kv_heads, head_dim))


def decode_fused(params: FusedParams) -> None:
    """One decode step of up to 8 single tokens as one persistent kernel (see decode_fused.cu).
    The caller fills ``params`` with device pointers and sizes; the launch is on the current stream."""
    _check(decode_fused_lib().ni_decode_fused(ctypes.byref(params), _stream()), "decode_fused")
